// selective.cuh -- device kernel of the selective scan of layered plans (B200_MIXER_ATTENTION_SCAN; its convolution is k_conv_rows).
// First user: Zulesun.
//
// Per channel c and state n, over the rows of a launch, S carried from launch to launch (zero at position 0):
//     dt = softplus(dt' + dt_bias[c]),   S[c][n] <- exp(-exp(A_log[c][n]) dt) S[c][n] + dt u[c] B[n],
//     y[c] = sum_n S[c][n] C[n] + D[c] u[c],   out[c] = out_scale * y[c] * silu(z[c])
//   * k_selective_scan<LPC, R>  LPC lanes share a channel, each keeps R of its states in registers; the rows of a launch run in sequence,
//                               channels in parallel over lanes and CTAs.  u, dt', z of the CTA's channels and B, C are staged TB tokens at a time
//                               with cp.async, double buffered; what needs no state (step size, step * u, gate) is worked out once per token and channel
//                               in a pass over the staged batch, so that the chain from token to token is one multiply-add.  Eight tokens'
//                               read-out sums are reduced together with seven shuffles.  A single-row launch computes dt' itself from its
//                               factor r and W_dt: the decode step has no launch of its own for that product.
// Everything is FP32 in both compute modes.
#pragma once
#include "delta.cuh"
#include "recurrent.cuh"

namespace ly {

struct SelScanArgs {
    int C, N, rank;        // channels, states per channel, entries of r in front of B and C in a parameter row
    const float *a2;       // [C][N]: -exp(A_log) * log2(e)
    const float *dt_bias, *D; // [C]
    const bf16 *w_dt;      // [C][rank] (single-row launches; nullptr: dt' is read from DT)
    float out_scale;
    int vec;               // 1: all row strides, column offsets, rank and N are multiples of 4 floats
};
#define SEL_THREADS 256
#define SEL_LANES 8
__host__ __device__ constexpr int sel_tb(int lpc, int) { return lpc >= 32 ? 8 : 16; } // tokens per staged batch
// States per lane when SEL_LANES lanes share a channel (up to 128 states), or a whole warp does; 0: more states than the kernel holds
__host__ __device__ inline int sel_reg_rows(int N) { return N <= 8 ? 1 : N <= 16 ? 2 : N <= 32 ? 4 : N <= 64 ? 8 : N <= 128 ? 16 : N <= 256 ? 8 : N <= 512 ? 16 : 0; }
__host__ __device__ inline int sel_lanes(int N) { return N <= 128 ? SEL_LANES : 32; }
__host__ __device__ inline size_t sel_state_floats(int C, int N) { return (size_t)C * sel_lanes(N) * sel_reg_rows(N); }
__host__ __device__ constexpr size_t sel_smem(int lpc, int r) { return (size_t)4 * sel_tb(lpc, r) * lpc * r * 4; }
// 2^x in one instruction (relative error 2^-22; results below the normal range are zero)
__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// R consecutive floats at p (16-byte aligned when R is a multiple of 4)
template <int R> __device__ __forceinline__ void load_run(const float *p, float (&v)[R]) {
    if constexpr (R % 4 == 0) {
#pragma unroll
        for (int i = 0; i < R; i += 4) { const float4 q = *reinterpret_cast<const float4 *>(p + i); v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w; }
    } else {
#pragma unroll
        for (int i = 0; i < R; i++) v[i] = p[i];
    }
}

// grid (ceil(C / (SEL_THREADS / LPC))), dynamic shared memory sel_smem(LPC, R).  U [n][ldu] convolved channels, PX [n][ldx] parameter rows [r | B | C], DT [n][lddt], Z [n][ldz].
// State: [channel][LPC * R] (states beyond N stay zero).  out32 / out16: row stride ldo, first column of this mixer.
template <int LPC, int R>
__global__ void __launch_bounds__(SEL_THREADS) k_selective_scan(const float *__restrict__ U, int ldu, const float *__restrict__ PX, int ldx, const float *__restrict__ DT, int lddt,
                                                                const float *__restrict__ Z, int ldz, SelScanArgs a, float *__restrict__ S, int n, const StepState *__restrict__ st,
                                                                float *__restrict__ out32, bf16 *__restrict__ out16, int ldo) {
    constexpr int CH = SEL_THREADS / LPC, RW = LPC * R, TB = sel_tb(LPC, R);
    __shared__ __align__(16) float us[2][TB][CH], ds[2][TB][CH], zs[2][TB][CH];
    typedef float Row[RW];
    extern __shared__ __align__(16) unsigned char selm[];
    Row *const Bs = reinterpret_cast<Row *>(selm), *const Cs = Bs + 2 * TB; // [buffer * TB + token]
    __shared__ float du[TB][CH], bs[CH], Dsm[CH];
    const int tid = threadIdx.x, l = tid % LPC, cl = tid / LPC, c0 = blockIdx.x * CH, c = c0 + cl;
    const bool live = c < a.C;
    const bool own_dt = a.w_dt != nullptr;
    auto fetch = [&](int t0, int buf) {
        const int nt = n - t0 < TB ? n - t0 : TB;
        if (a.vec) {
            for (int e = tid; e < TB * (CH / 4); e += SEL_THREADS) {
                const int t = e / (CH / 4), i = (e % (CH / 4)) * 4;
                const bool ok = t < nt && c0 + i < a.C; // a.C is a multiple of 4 here
                const size_t tt = ok ? t0 + t : 0;
                cp_async16(&us[buf][t][i], ok ? U + tt * ldu + c0 + i : U, ok);
                cp_async16(&zs[buf][t][i], ok ? Z + tt * ldz + c0 + i : Z, ok);
                if (!own_dt) cp_async16(&ds[buf][t][i], ok ? DT + tt * lddt + c0 + i : DT, ok);
            }
            for (int e = tid; e < TB * (RW / 4); e += SEL_THREADS) {
                const int t = e / (RW / 4), i = (e % (RW / 4)) * 4;
                const bool ok = t < nt && i < a.N;
                const float *p = PX + (size_t)(ok ? t0 + t : 0) * ldx + a.rank;
                cp_async16(&Bs[buf * TB + t][i], ok ? p + i : PX, ok);
                cp_async16(&Cs[buf * TB + t][i], ok ? p + a.N + i : PX, ok);
            }
        } else {
            for (int e = tid; e < TB * CH; e += SEL_THREADS) {
                const int t = e / CH, i = e % CH;
                const bool ok = t < nt && c0 + i < a.C;
                const size_t tt = ok ? t0 + t : 0;
                cp_async4(&us[buf][t][i], ok ? U + tt * ldu + c0 + i : U, ok);
                cp_async4(&zs[buf][t][i], ok ? Z + tt * ldz + c0 + i : Z, ok);
                if (!own_dt) cp_async4(&ds[buf][t][i], ok ? DT + tt * lddt + c0 + i : DT, ok);
            }
            for (int e = tid; e < TB * RW; e += SEL_THREADS) {
                const int t = e / RW, i = e % RW;
                const bool ok = t < nt && i < a.N;
                const float *p = PX + (size_t)(ok ? t0 + t : 0) * ldx + a.rank;
                cp_async4(&Bs[buf * TB + t][i], ok ? p + i : PX, ok);
                cp_async4(&Cs[buf * TB + t][i], ok ? p + a.N + i : PX, ok);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    float s[R], A[R];
    const bool fresh = st->pos == 0;
    float *Sg = S + (size_t)c * RW + l * R;
    if (live && !fresh) load_run<R>(Sg, s);
    else {
#pragma unroll
        for (int i = 0; i < R; i++) s[i] = 0.0f;
    }
#pragma unroll
    for (int i = 0; i < R; i++) A[i] = live && l * R + i < a.N ? a.a2[(size_t)c * a.N + l * R + i] : 0.0f;
    if (tid < CH) { bs[tid] = c0 + tid < a.C ? a.dt_bias[c0 + tid] : 0.0f; Dsm[tid] = c0 + tid < a.C ? a.D[c0 + tid] : 0.0f; }
    if (own_dt) { // dt' of the only row: a warp per channel, W_dt streamed
        const int lane = tid & 31, warp = tid >> 5;
        const bool vec = (a.rank & 7) == 0 && (((size_t)a.w_dt) & 15) == 0 && (((size_t)PX) & 15) == 0;
#pragma unroll 4
        for (int k = warp; k < CH; k += SEL_THREADS / 32) {
            if (c0 + k >= a.C) break;
            const float v = dot_row_bf16(a.w_dt + (size_t)(c0 + k) * a.rank, PX, a.rank, lane, vec);
            if (lane == 0) ds[0][0][k] = v;
        }
    }
    int buf = 0;
    const int q = l & 7;
    for (int t0 = 0; t0 < n; t0 += TB, buf ^= 1) {
        const int nt = n - t0 < TB ? n - t0 : TB;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads(); // this batch has landed for every thread, and the other buffer's batch is consumed
        if (t0 + TB < n) fetch(t0 + TB, buf ^ 1);
        // per token and channel: step size, step * u, D * u, gate; a token behind the last gets step 0 and leaves the state as it is
#pragma unroll
        for (int e = tid; e < TB * CH; e += SEL_THREADS) {
            const int t = e / CH, i = e % CH;
            const float u = us[buf][t][i], z = zs[buf][t][i];
            const float dt = t < nt ? softplusf_(ds[buf][t][i] + bs[i]) : 0.0f;
            ds[buf][t][i] = dt;
            us[buf][t][i] = dt * u;
            du[t][i] = Dsm[i] * u;
            zs[buf][t][i] = z / (1.0f + expf(-z)) * a.out_scale;
        }
        __syncthreads();
#pragma unroll
        for (int tb = 0; tb < TB; tb += 8) {
            if (tb >= nt) break;
            float acc[8];
#pragma unroll
            for (int k = 0; k < 8; k++) {
                const float dt = ds[buf][tb + k][cl], dx = us[buf][tb + k][cl];
                float bv[R], cv[R];
                load_run<R>(&Bs[buf * TB + tb + k][l * R], bv);
                load_run<R>(&Cs[buf * TB + tb + k][l * R], cv);
                float ac = 0.0f;
#pragma unroll
                for (int i = 0; i < R; i++) {
                    s[i] = fmaf(exp2_approx(dt * A[i]), s[i], dx * bv[i]);
                    ac = fmaf(s[i], cv[i], ac);
                }
                acc[k] = ac;
            }
            const bool h4 = q & 4, h2 = q & 2, h1 = q & 1; // lane q of every eight ends up with the sum of token tb + q
            float p4[4], p2[2];
#pragma unroll
            for (int k = 0; k < 4; k++) p4[k] = (h4 ? acc[k + 4] : acc[k]) + __shfl_xor_sync(0xffffffffu, h4 ? acc[k] : acc[k + 4], 4);
#pragma unroll
            for (int k = 0; k < 2; k++) p2[k] = (h2 ? p4[k + 2] : p4[k]) + __shfl_xor_sync(0xffffffffu, h2 ? p4[k] : p4[k + 2], 2);
            float v = (h1 ? p2[1] : p2[0]) + __shfl_xor_sync(0xffffffffu, h1 ? p2[0] : p2[1], 1);
#pragma unroll
            for (int o = 8; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (tb + q < nt && live && l < 8) {
                const float o = (v + du[tb + q][cl]) * zs[buf][tb + q][cl];
                const size_t at = (size_t)(t0 + tb + q) * ldo + c;
                if (out32) out32[at] = o;
                if (out16) out16[at] = __float2bfloat16_rn(o);
            }
        }
    }
    if (live) {
        if constexpr (R % 4 == 0) {
#pragma unroll
            for (int i = 0; i < R; i += 4) *reinterpret_cast<float4 *>(Sg + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
        } else {
#pragma unroll
            for (int i = 0; i < R; i++) Sg[i] = s[i];
        }
    }
}

} // namespace ly
