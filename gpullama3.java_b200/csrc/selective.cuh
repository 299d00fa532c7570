// selective.cuh -- device kernel of the selective scan of layered plans (B200_MIXER_ATTENTION_SCAN; its convolution is k_conv_rows).
// First user: Zulesun.
//
// Per channel c and state n, over the rows of a launch, S carried from launch to launch (zero at position 0):
//     dt = softplus(dt' + dt_bias[c]),   S[c][n] <- exp(-exp(A_log[c][n]) dt) S[c][n] + dt u[c] B[n],
//     y[c] = sum_n S[c][n] C[n] + D[c] u[c],   out[c] = out_scale * y[c] * silu(z[c])
//   * k_selective_scan<LPC, R>  LPC lanes share a channel, each keeps R of its states in registers (packed pairs: one instruction works on two); the
//                               rows of a launch run in sequence, channels in parallel over lanes and CTAs.  u, dt', z of the CTA's channels and B, C
//                               travel to shared memory TB tokens at a time with cp.async, three batches ahead.  The warps have two roles: four
//                               of them fetch, and work out what needs no state (step size, step * u, gate, D u * gate) once per token and
//                               channel, for the next batch while the other four scan the current one; the chain from token to token is one
//                               multiply-add, and a batch costs one barrier.  Four tokens' exponentials are in flight together, and their
//                               read-out sums are reduced with three shuffles.  A single-row launch computes dt' itself from its factor r and
//                               W_dt: the decode step has no launch of its own for that product.
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
#define SEL_THREADS 128              // threads of each role
#define SEL_BLOCK (2 * SEL_THREADS)
#define SEL_LANES 4
#define SEL_BUFS 4
__host__ __device__ constexpr int sel_tb(int lpc) { return lpc >= 32 ? 8 : 16; } // tokens per staged batch
// States per lane when SEL_LANES lanes share a channel (up to 128 states), or a whole warp does; 0: more states than the kernel holds
__host__ __device__ inline int sel_reg_rows(int N) { return N <= 4 ? 1 : N <= 8 ? 2 : N <= 16 ? 4 : N <= 32 ? 8 : N <= 64 ? 16 : N <= 128 ? 32 : N <= 256 ? 8 : N <= 512 ? 16 : 0; }
__host__ __device__ inline int sel_lanes(int N) { return N <= 128 ? SEL_LANES : 32; }
__host__ __device__ inline size_t sel_state_floats(int C, int N) { return (size_t)C * sel_lanes(N) * sel_reg_rows(N); }
// staged u, dt', z and B, C of SEL_BUFS batches, the worked-out four numbers per token and channel of two
__host__ __device__ constexpr size_t sel_smem(int lpc, int r) { return (size_t)sel_tb(lpc) * 4 * (SEL_BUFS * (3 * (SEL_THREADS / lpc) + 2 * lpc * r) + 2 * 4 * (SEL_THREADS / lpc)); }

// 2^x in one instruction (relative error 2^-22; results below the normal range are zero)
__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// log(1 + e^x) without the branches of a general logarithm: max(x, 0) + log1p(t), t = e^-|x| in (0, 1], and log1p(t) = 2 artanh(w), w = t / (2 + t) <= 1/3,
// by the first eight terms of artanh's power series (the ninth is below 2e-9 of the first)
__device__ __forceinline__ float softplus_series(float x) {
    const float t = expf(-fabsf(x)), w = __fdividef(t, 2.0f + t), z = w * w;
    float p = 1.0f / 15.0f;
    p = fmaf(p, z, 1.0f / 13.0f);
    p = fmaf(p, z, 1.0f / 11.0f);
    p = fmaf(p, z, 1.0f / 9.0f);
    p = fmaf(p, z, 1.0f / 7.0f);
    p = fmaf(p, z, 1.0f / 5.0f);
    p = fmaf(p, z, 1.0f / 3.0f);
    p = fmaf(p, z, 1.0f);
    return fmaf(2.0f * w, p, fmaxf(x, 0.0f));
}
// Two FP32 operations in one instruction, each rounded as usual
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("{\n.reg .b64 a, b, d;\nmov.b64 a, {%2, %3};\nmov.b64 b, {%4, %5};\nmul.rn.f32x2 d, a, b;\nmov.b64 {%0, %1}, d;\n}" : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("{\n.reg .b64 a, b, c, d;\nmov.b64 a, {%2, %3};\nmov.b64 b, {%4, %5};\nmov.b64 c, {%6, %7};\nfma.rn.f32x2 d, a, b, c;\nmov.b64 {%0, %1}, d;\n}"
        : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
    return d;
}
// R consecutive floats at p (16-byte aligned when R is a multiple of 4, 8-byte when it is 2) as pairs (R = 1: one half pair)
template <int R> __device__ __forceinline__ void load_pairs(const float *p, float2 (&v)[(R + 1) / 2]) {
    if constexpr (R % 4 == 0) {
#pragma unroll
        for (int i = 0; i < R; i += 4) { const float4 q = *reinterpret_cast<const float4 *>(p + i); v[i / 2] = make_float2(q.x, q.y); v[i / 2 + 1] = make_float2(q.z, q.w); }
    } else if constexpr (R == 2) v[0] = *reinterpret_cast<const float2 *>(p);
    else v[0] = make_float2(p[0], 0.0f);
}

// grid (ceil(C / (SEL_THREADS / LPC))), dynamic shared memory sel_smem(LPC, R).  U [n][ldu] convolved channels, PX [n][ldx] parameter rows [r | B | C], DT [n][lddt],
// Z [n][ldz].  State: [channel][LPC * R] (states beyond N stay zero).  out32 / out16: row stride ldo, first column of this mixer.
template <int LPC, int R>
__global__ void __launch_bounds__(SEL_BLOCK) k_selective_scan(const float *__restrict__ U, int ldu, const float *__restrict__ PX, int ldx, const float *__restrict__ DT, int lddt,
                                                                const float *__restrict__ Z, int ldz, SelScanArgs a, float *__restrict__ S, int n, const StepState *__restrict__ st,
                                                                float *__restrict__ out32, bf16 *__restrict__ out16, int ldo) {
    constexpr int CH = SEL_THREADS / LPC, RW = LPC * R, TB = sel_tb(LPC), RP = (R + 1) / 2;
    extern __shared__ __align__(16) float selm[];
    typedef float CRow[CH];
    typedef float SRow[RW];
    typedef float4 PRow[CH];
    PRow *const prep = reinterpret_cast<PRow *>(selm);                       // [2 * TB]: {dt, dt u, gate, D u gate}
    SRow *const Bs = reinterpret_cast<SRow *>(prep + 2 * TB), *const Cs = Bs + SEL_BUFS * TB; // [buffer * TB + token]
    CRow *const us = reinterpret_cast<CRow *>(Cs + SEL_BUFS * TB), *const ds = us + SEL_BUFS * TB, *const zs = ds + SEL_BUFS * TB;
    __shared__ float bs[CH], Dsm[CH];
    const bool scans = threadIdx.x < SEL_THREADS; // role: warps 0 .. 3 scan, 4 .. 7 fetch and work out (tid counts within a role)
    const int tid = threadIdx.x % SEL_THREADS, l = tid % LPC, cl = tid / LPC, c0 = blockIdx.x * CH, c = c0 + cl;
    const bool live = c < a.C, own_dt = a.w_dt != nullptr;
    const int batches = (n + TB - 1) / TB;
    auto fetch = [&](int b) { // every call commits a group, also past the last batch
        if (b < batches) {
            const int t0 = b * TB, nt = n - t0 < TB ? n - t0 : TB, at = b % SEL_BUFS * TB;
            if (a.vec) {
                for (int e = tid; e < TB * (CH / 4); e += SEL_THREADS) {
                    const int t = e / (CH / 4), i = (e % (CH / 4)) * 4;
                    const bool ok = t < nt && c0 + i < a.C; // a.C is a multiple of 4 here
                    const size_t tt = ok ? t0 + t : 0;
                    cp_async16(&us[at + t][i], ok ? U + tt * ldu + c0 + i : U, ok);
                    cp_async16(&zs[at + t][i], ok ? Z + tt * ldz + c0 + i : Z, ok);
                    if (!own_dt) cp_async16(&ds[at + t][i], ok ? DT + tt * lddt + c0 + i : DT, ok);
                }
                for (int e = tid; e < TB * (RW / 4); e += SEL_THREADS) {
                    const int t = e / (RW / 4), i = (e % (RW / 4)) * 4;
                    const bool ok = t < nt && i < a.N;
                    const float *p = PX + (size_t)(ok ? t0 + t : 0) * ldx + a.rank;
                    cp_async16(&Bs[at + t][i], ok ? p + i : PX, ok);
                    cp_async16(&Cs[at + t][i], ok ? p + a.N + i : PX, ok);
                }
            } else {
                for (int e = tid; e < TB * CH; e += SEL_THREADS) {
                    const int t = e / CH, i = e % CH;
                    const bool ok = t < nt && c0 + i < a.C;
                    const size_t tt = ok ? t0 + t : 0;
                    cp_async4(&us[at + t][i], ok ? U + tt * ldu + c0 + i : U, ok);
                    cp_async4(&zs[at + t][i], ok ? Z + tt * ldz + c0 + i : Z, ok);
                    if (!own_dt) cp_async4(&ds[at + t][i], ok ? DT + tt * lddt + c0 + i : DT, ok);
                }
                for (int e = tid; e < TB * RW; e += SEL_THREADS) {
                    const int t = e / RW, i = e % RW;
                    const bool ok = t < nt && i < a.N;
                    const float *p = PX + (size_t)(ok ? t0 + t : 0) * ldx + a.rank;
                    cp_async4(&Bs[at + t][i], ok ? p + i : PX, ok);
                    cp_async4(&Cs[at + t][i], ok ? p + a.N + i : PX, ok);
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // per token and channel of batch b: step size, step * u, gate, D u * gate; a token behind the last gets step 0 and leaves the state as it is
    auto work_out = [&](int b) {
        if (b >= batches) return;
        const int nt = n - b * TB, at = b % SEL_BUFS * TB, to = (b & 1) * TB;
        constexpr int PER = TB * CH / SEL_THREADS > 0 ? TB * CH / SEL_THREADS : 1;
        float u[PER], z[PER], d[PER];
        float4 w[PER];
#pragma unroll
        for (int k = 0; k < PER; k++) {
            const int e = tid + k * SEL_THREADS, t = e / CH, i = e % CH;
            if (e >= TB * CH) continue;
            u[k] = us[at + t][i]; z[k] = zs[at + t][i]; d[k] = ds[at + t][i] + bs[i];
        }
#pragma unroll
        for (int k = 0; k < PER; k++) {
            const int e = tid + k * SEL_THREADS, t = e / CH, i = e % CH;
            if (e >= TB * CH) continue;
            const float dt = t < nt ? softplus_series(d[k]) : 0.0f, g = z[k] * sigmoid_fast(z[k]) * a.out_scale;
            w[k] = make_float4(dt, dt * u[k], g, Dsm[i] * u[k] * g);
        }
#pragma unroll
        for (int k = 0; k < PER; k++) {
            const int e = tid + k * SEL_THREADS;
            if (e < TB * CH) prep[to + e / CH][e % CH] = w[k];
        }
    };
    if (!scans) for (int b = 0; b < SEL_BUFS - 1; b++) fetch(b);
    for (int i = threadIdx.x; i < CH; i += SEL_BLOCK) { bs[i] = c0 + i < a.C ? a.dt_bias[c0 + i] : 0.0f; Dsm[i] = c0 + i < a.C ? a.D[c0 + i] : 0.0f; }
    float2 s[RP], A[RP];
    const bool fresh = st->pos == 0;
    float *Sg = S + (size_t)c * RW + l * R;
    if (scans && live && !fresh) load_pairs<R>(Sg, s);
    else {
#pragma unroll
        for (int i = 0; i < RP; i++) s[i] = make_float2(0.0f, 0.0f);
    }
    auto exponent = [&](int i) { return i < R && scans && live && l * R + i < a.N ? a.a2[(size_t)c * a.N + l * R + i] : 0.0f; };
#pragma unroll
    for (int i = 0; i < RP; i++) A[i] = make_float2(exponent(2 * i), exponent(2 * i + 1));
    if (own_dt) { // dt' of the only row: a warp per channel, W_dt streamed
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        const bool vec = (a.rank & 7) == 0 && (((size_t)a.w_dt) & 15) == 0 && (((size_t)PX) & 15) == 0;
#pragma unroll 4
        for (int k = warp; k < CH; k += SEL_BLOCK / 32) {
            if (c0 + k >= a.C) break;
            const float v = dot_row_bf16(a.w_dt + (size_t)(c0 + k) * a.rank, PX, a.rank, lane, vec);
            if (lane == 0) ds[0][k] = v;
        }
    }
    asm volatile("cp.async.wait_group %0;" ::"n"(SEL_BUFS - 2) : "memory"); // the first batch has landed (the scanning threads have no copies of their own)
    __syncthreads();
    if (!scans) work_out(0);
    const int q = l & 3;
    for (int b = 0; b < batches; b++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(SEL_BUFS - 3) : "memory"); // batch b + 1 has landed
        __syncthreads(); // batch b is worked out, batch b - 1 consumed
        if (!scans) {
            fetch(b + SEL_BUFS - 1);
            work_out(b + 1);
            continue;
        }
        const int t0 = b * TB, nt = n - t0 < TB ? n - t0 : TB, at = b % SEL_BUFS * TB;
        const PRow *const P = prep + (b & 1) * TB;
        auto four = [&](int tb) { // tokens tb .. tb + 3 of the batch
            constexpr int G = R <= 8 ? 4 : 1; // tokens whose operands and exponentials are fetched ahead of the chain
            float acc[4];
#pragma unroll
            for (int k0 = 0; k0 < 4; k0 += G) {
                float2 e[G][RP], db[G][RP], cv[G][RP];
#pragma unroll
                for (int k = 0; k < G; k++) {
                    const float2 p = *reinterpret_cast<const float2 *>(&P[tb + k0 + k][cl]);
                    load_pairs<R>(&Bs[at + tb + k0 + k][l * R], db[k]);
                    load_pairs<R>(&Cs[at + tb + k0 + k][l * R], cv[k]);
#pragma unroll
                    for (int i = 0; i < RP; i++) {
                        e[k][i] = mul2(make_float2(p.x, p.x), A[i]);
                        db[k][i] = mul2(make_float2(p.y, p.y), db[k][i]);
                    }
                }
#pragma unroll
                for (int k = 0; k < G; k++)
#pragma unroll
                    for (int i = 0; i < RP; i++) e[k][i] = make_float2(exp2_approx(e[k][i].x), exp2_approx(e[k][i].y));
#pragma unroll
                for (int k = 0; k < G; k++) {
                    float2 ac = make_float2(0.0f, 0.0f);
#pragma unroll
                    for (int i = 0; i < RP; i++) {
                        s[i] = fma2(e[k][i], s[i], db[k][i]);
                        ac = fma2(s[i], cv[k][i], ac);
                    }
                    acc[k0 + k] = ac.x + ac.y;
                }
            }
            const bool h2 = q & 2, h1 = q & 1; // lane q of every four ends up with the sum of token tb + q
            float p0 = h2 ? acc[2] : acc[0], p1 = h2 ? acc[3] : acc[1];
            p0 += __shfl_xor_sync(0xffffffffu, h2 ? acc[0] : acc[2], 2);
            p1 += __shfl_xor_sync(0xffffffffu, h2 ? acc[1] : acc[3], 2);
            float v = (h1 ? p1 : p0) + __shfl_xor_sync(0xffffffffu, h1 ? p0 : p1, 1);
#pragma unroll
            for (int o = 4; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (tb + q < nt && live && l < 4) {
                const float4 w = P[tb + q][cl];
                const float o = fmaf(v, w.z, w.w);
                const size_t to = (size_t)(t0 + tb + q) * ldo + c;
                if (out32) out32[to] = o;
                if (out16) out16[to] = __float2bfloat16_rn(o);
            }
        };
        four(0);
        if (nt > 4) { // without a branch between the groups, so that their independent parts overlap
#pragma unroll
            for (int tb = 4; tb < TB; tb += 4) four(tb);
        }
    }
    if (!scans || !live) return;
    if constexpr (R % 4 == 0) {
#pragma unroll
        for (int i = 0; i < RP; i += 2) *reinterpret_cast<float4 *>(Sg + 2 * i) = make_float4(s[i].x, s[i].y, s[i + 1].x, s[i + 1].y);
    } else if constexpr (R == 2) *reinterpret_cast<float2 *>(Sg) = s[0];
    else Sg[0] = s[0].x;
}

} // namespace ly
