// Mamba, the selective scan: a recurrent mixer with `state_size` numbers per channel, each with a decay of its own per token (libktb200_seq.so).
//
//   dt = softplus(dt_logit + dt_bias_c) ;  S_cn <- exp(dt a_cn) S_cn + dt x_c B_n ;  y_c = sum_n S_cn C_n + D_c x_c ;  out_c = y_c silu(z_c)
//
//   ktb200_selective_scan   prompt portions and decode steps alike, one launch (its x: ktb200_conv_silu, csrc/ssd.cu)
//
// State row of a sequence and layer (fp32): [ S inner x state_size | filter inputs (taps - 1) x inner, oldest first ], read from the row seqs[2][s] (or
// zeros when -1) and written to the row seqs[3][s].  Storage type T (bf16 or float) for projections, the filtered channels and the output; steps,
// decays, the state and everything read from it are fp32.
#include <cuda_bf16.h>

#include "common.cuh"
#include "seq_common.cuh"

namespace ktb {

struct SelScan {
    const void *x, *dt, *B, *C, *z;
    long dt_stride, bc_stride, z_stride;
    const float *dt_bias, *A, *D;
    int inner, N;
    const int* seqs;
    int seqs_stride;
    float* state;
    long state_stride;
    int vec_state;
};

// S exp(dt a) + u.  Where activations are bf16: one base-2 exponential of a factor scaled once per thread.  In 32-bit runs the factor is taken as
// 1 + expm1(dt a): slow channels (factors just below one) would otherwise lose the same part of an ulp with every token.
template <typename T> __device__ __forceinline__ float decay_factor(float a);
template <> __device__ __forceinline__ float decay_factor<float>(float a) { return a; }
template <> __device__ __forceinline__ float decay_factor<__nv_bfloat16>(float a) { return a * 1.4426950408889634f; }
template <typename T> __device__ __forceinline__ float decayed(float S, float dt, float f, float u);
template <> __device__ __forceinline__ float decayed<float>(float S, float dt, float f, float u) { return fmaf(expm1f(dt * f), S, S) + u; }
template <> __device__ __forceinline__ float decayed<__nv_bfloat16>(float S, float dt, float f, float u) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(dt * f));
    return fmaf(r, S, u);
}

// grid (channel blocks, portions), 128 threads: L neighbouring lanes share a channel, SPT states each, in registers.  Tokens run in order in chunks of
// TC, whose dt (after the softplus), x, B and C sit in shared memory; the next chunk's inputs are fetched into registers meanwhile.  Four tokens'
// parts of y at a time are added over the lanes of a channel so that every shuffle halves the tokens a lane still holds.
template <typename T, int SPT, int L>
__global__ void __launch_bounds__(128) selective_scan_kernel(const SelScan a, T* __restrict__ out) {
    constexpr int CH = 128 / L, CP = CH + 8, NP = SPT * L, TC = NP <= 64 ? 16 : 8;
    constexpr int E = TC * CH >= 128 ? TC * CH / 128 : 1, EB = TC * NP >= 128 ? TC * NP / 128 : 1;
    __shared__ float dts[TC * CH], xs[TC * CH], ys[TC * CP];
    __shared__ __align__(16) float Bs[TC * NP];
    __shared__ __align__(16) float Cs[TC * NP];
    const int tid = threadIdx.x, l = tid % L, ch = tid / L, ch0 = blockIdx.x * CH, s = blockIdx.y, N = a.N, inner = a.inner;
    const int start = a.seqs[s], len = a.seqs[a.seqs_stride + s], rd = a.seqs[2 * a.seqs_stride + s], wr = a.seqs[3 * a.seqs_stride + s];
    const bool live = ch0 + ch < inner;
    const long at = (long)(ch0 + ch) * N + l * SPT;
    float S[SPT], f[SPT];
#pragma unroll
    for (int k = 0; k < SPT; k++) S[k] = f[k] = 0.f;
    if (live && a.vec_state) {
#pragma unroll
        for (int k = 0; k < SPT; k += 4) {
            if (l * SPT + k < N) {
                const float4 w = load4(a.A + at + k);
                f[k] = w.x; f[k + 1] = w.y; f[k + 2] = w.z; f[k + 3] = w.w;
                if (rd >= 0) {
                    const float4 u = load4(a.state + (long)rd * a.state_stride + at + k);
                    S[k] = u.x; S[k + 1] = u.y; S[k + 2] = u.z; S[k + 3] = u.w;
                }
            }
        }
    } else if (live) {
#pragma unroll
        for (int k = 0; k < SPT; k++) {
            if (l * SPT + k < N) {
                f[k] = a.A[at + k];
                if (rd >= 0) S[k] = a.state[(long)rd * a.state_stride + at + k];
            }
        }
    }
#pragma unroll
    for (int k = 0; k < SPT; k++) f[k] = decay_factor<T>(f[k]);
    // staging: this thread's channel is tid % CH for every token it fetches
    const int sc = ch0 + tid % CH;
    const bool sok = sc < inner;
    const float bias = sok ? a.dt_bias[sc] : 0.f, skip = sok ? a.D[sc] : 0.f;
    float rx[E], rdt[E], rz[E], rb[EB], rc[EB];
    auto fetch = [&](int t0) {
        const int nt = min(TC, len - t0);
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = e * 128 + tid, tt = i / CH;
            rx[e] = rdt[e] = rz[e] = 0.f;
            if (tt < nt && sok) {
                const long t = start + t0 + tt;
                rx[e] = to_f(((const T*)a.x)[t * inner + sc]);
                rdt[e] = to_f(((const T*)a.dt)[t * a.dt_stride + sc]);
                rz[e] = to_f(((const T*)a.z)[t * a.z_stride + sc]);
            }
        }
#pragma unroll
        for (int e = 0; e < EB; e++) {
            const int i = e * 128 + tid, tt = i / NP, n = i % NP;
            rb[e] = rc[e] = 0.f;
            if (tt < nt && n < N) {
                const long t = start + t0 + tt;
                rb[e] = to_f(((const T*)a.B)[t * a.bc_stride + n]);
                rc[e] = to_f(((const T*)a.C)[t * a.bc_stride + n]);
            }
        }
    };
    if (len > 0) fetch(0);
    for (int t0 = 0; t0 < len; t0 += TC) {
        const int nt = min(TC, len - t0);
        float cx[E], cz[E];
        __syncthreads();      // the previous chunk is consumed
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = e * 128 + tid, tt = i / CH;
            cx[e] = rx[e];
            cz[e] = rz[e];
            if (i < TC * CH) {
                const float v = rdt[e] + bias;
                xs[i] = rx[e];
                dts[i] = tt < nt ? (v > 20.f ? v : log1pf(expf(v))) : 0.f;      // (a padding token leaves the state alone)
            }
        }
#pragma unroll
        for (int e = 0; e < EB; e++) {
            const int i = e * 128 + tid;
            if (i < TC * NP) { Bs[i] = rb[e]; Cs[i] = rc[e]; }
        }
        __syncthreads();
        if (t0 + TC < len) fetch(t0 + TC);
        for (int tg = 0; tg < nt; tg += 4) {
            float y[4];
#pragma unroll
            for (int q = 0; q < 4; q++) {
                const int tt = tg + q;
                const float dt = dts[tt * CH + ch], dx = dt * xs[tt * CH + ch];
                y[q] = 0.f;
#pragma unroll
                for (int k = 0; k < SPT; k += 4) {
                    const float4 b = load4(Bs + tt * NP + l * SPT + k), c = load4(Cs + tt * NP + l * SPT + k);
                    S[k] = decayed<T>(S[k], dt, f[k], dx * b.x);
                    y[q] = fmaf(S[k], c.x, y[q]);
                    S[k + 1] = decayed<T>(S[k + 1], dt, f[k + 1], dx * b.y);
                    y[q] = fmaf(S[k + 1], c.y, y[q]);
                    S[k + 2] = decayed<T>(S[k + 2], dt, f[k + 2], dx * b.z);
                    y[q] = fmaf(S[k + 2], c.z, y[q]);
                    S[k + 3] = decayed<T>(S[k + 3], dt, f[k + 3], dx * b.w);
                    y[q] = fmaf(S[k + 3], c.w, y[q]);
                }
            }
            if (L == 1) {
#pragma unroll
                for (int q = 0; q < 4; q++) ys[(tg + q) * CP + ch] = y[q];
            } else {      // lane bit 0 keeps tokens {0, 1} or {2, 3}, lane bit 1 one of the two
                const bool b0 = l & 1, b1 = l & 2;
                float k0 = b0 ? y[2] : y[0], k1 = b0 ? y[3] : y[1];
                k0 += __shfl_xor_sync(0xffffffffu, b0 ? y[0] : y[2], 1);
                k1 += __shfl_xor_sync(0xffffffffu, b0 ? y[1] : y[3], 1);
                if (L == 2) {
                    ys[(tg + 2 * b0) * CP + ch] = k0;
                    ys[(tg + 2 * b0 + 1) * CP + ch] = k1;
                } else {
                    float v = b1 ? k1 : k0;
                    v += __shfl_xor_sync(0xffffffffu, b1 ? k0 : k1, 2);
#pragma unroll
                    for (int o = 4; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                    if (l < 4) ys[(tg + 2 * b0 + b1) * CP + ch] = v;
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = e * 128 + tid, tt = i / CH;
            if (tt < nt && sok) out[(long)(start + t0 + tt) * inner + sc] = from_f<T>(fmaf(skip, cx[e], ys[tt * CP + tid % CH]) * act_silu(cz[e]));
        }
    }
    if (wr >= 0 && live) {
        float* w = a.state + (long)wr * a.state_stride + at;
#pragma unroll
        for (int k = 0; k < SPT; k += 4) {
            if (a.vec_state) {
                if (l * SPT + k < N) store4(w + k, make_float4(S[k], S[k + 1], S[k + 2], S[k + 3]));
            } else {
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (l * SPT + k + e < N) w[k + e] = S[k + e];
            }
        }
    }
}

}  // namespace ktb

using namespace ktb;

#define SEQ_DISPATCH(dtype, ...)                                                           \
    do {                                                                                   \
        if ((dtype) == KTB200_TYPE_BF16) { using T = __nv_bfloat16; __VA_ARGS__; }         \
        else if ((dtype) == KTB200_TYPE_F32) { using T = float; __VA_ARGS__; }             \
        else { set_error("dtype must be bf16 or f32"); return KTB200_EINVAL; }             \
    } while (0)

extern "C" int ktb200_selective_scan(const ktb200_selective_scan_params* c, void* out, int dtype, void* stream) {
    if (!c || !c->x || !c->dt_logit || !c->b || !c->c || !c->z || !c->dt_bias || !c->a || !c->d_skip || !c->seqs || !c->state || !out || c->inner <= 0 || c->state_size <= 0 ||
        c->state_size > 256) {
        set_error("selective_scan: bad argument (state size <= 256)");
        return KTB200_EINVAL;
    }
    if (c->n_seqs <= 0) return KTB200_OK;
    const int N = c->state_size;
    auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const SelScan a{c->x, c->dt_logit, c->b, c->c, c->z, c->dt_stride, c->bc_stride, c->z_stride, c->dt_bias, c->a, c->d_skip, c->inner, N, c->seqs, c->seqs_stride, c->state,
                    c->state_stride, N % 4 == 0 && c->state_stride % 4 == 0 && al(c->state) && al(c->a)};
#define SCAN_LAUNCH(SPT, L) \
    SEQ_DISPATCH(dtype, { selective_scan_kernel<T, SPT, L><<<dim3((c->inner + 128 / (L) - 1) / (128 / (L)), c->n_seqs), 128, 0, (cudaStream_t)stream>>>(a, (T*)out); })
    if (N <= 4) SCAN_LAUNCH(4, 1);
    else if (N <= 8) SCAN_LAUNCH(4, 2);
    else if (N <= 16) SCAN_LAUNCH(4, 4);
    else if (N <= 32) SCAN_LAUNCH(4, 8);
    else if (N <= 64) SCAN_LAUNCH(4, 16);
    else if (N <= 128) SCAN_LAUNCH(4, 32);
    else SCAN_LAUNCH(8, 32);
#undef SCAN_LAUNCH
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}
