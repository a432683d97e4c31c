// Mamba, the selective scan: a recurrent mixer with `state_size` numbers per channel, each with a decay of its own per token (libktb200_seq.so).
//
//   dt = softplus(dt_logit + dt_bias_c) ;  S_cn <- exp(dt a_cn) S_cn + dt x_c B_n ;  y_c = sum_n S_cn C_n + D_c x_c ;  out_c = y_c silu(z_c)
//
//   ktb200_selective_scan   steps, recurrence, skip and gate of prompt portions or of decode steps in one launch (its x: ktb200_conv_silu, csrc/ssd.cu)
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

// Two neighbouring states at a time.  Where activations are bf16, on the packed fp32 pipe: the factors a come scaled by log2(e), a decay is one base-2
// exponential.  In 32-bit runs the decay is taken as 1 + expm1(dt a): slow channels (factors just below one) would otherwise lose the same part
// of an ulp with every token.
__device__ __forceinline__ uint64_t pair_of(float x, float y) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
    return r;
}
__device__ __forceinline__ float2 halves_of(uint64_t v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ uint64_t mul_pairs(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ uint64_t fma_pairs(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
template <typename T> struct ScanMath;
template <> struct ScanMath<__nv_bfloat16> {
    static __device__ __forceinline__ float factor(float a) { return a * 1.4426950408889634f; }
    // S <- exp(dt a) S + dx B ;  y += S C
    static __device__ __forceinline__ void step(uint64_t& S, uint64_t f, float dt, float dx, float2 b, float2 c, uint64_t& y) {
        const float2 e = halves_of(mul_pairs(pair_of(dt, dt), f));
        S = fma_pairs(pair_of(exp2_approx(e.x), exp2_approx(e.y)), S, mul_pairs(pair_of(dx, dx), pair_of(b.x, b.y)));
        y = fma_pairs(S, pair_of(c.x, c.y), y);
    }
    // max(x, 0) + log(1 + u), u = exp(-|x|): log(1 + u) = 2 artanh(s) with s = u / (2 + u) <= 1/3, by its power series (the first term left out is below 1e-9 of the sum)
    static __device__ __forceinline__ float softplus(float x) {
        const float u = exp2_approx(-1.4426950408889634f * fabsf(x)), s = __fdividef(u, 2.0f + u), q = s * s;
        float p = 1.0f / 17.0f;
        p = fmaf(p, q, 1.0f / 15.0f);
        p = fmaf(p, q, 1.0f / 13.0f);
        p = fmaf(p, q, 1.0f / 11.0f);
        p = fmaf(p, q, 1.0f / 9.0f);
        p = fmaf(p, q, 1.0f / 7.0f);
        p = fmaf(p, q, 0.2f);
        p = fmaf(p, q, 1.0f / 3.0f);
        return fmaxf(x, 0.f) + 2.0f * fmaf(p * q, s, s);
    }
};
template <> struct ScanMath<float> {
    static __device__ __forceinline__ float factor(float a) { return a; }
    static __device__ __forceinline__ void step(uint64_t& S, uint64_t f, float dt, float dx, float2 b, float2 c, uint64_t& y) {
        float2 s = halves_of(S), o = halves_of(y);
        const float2 a = halves_of(f);
        s.x = fmaf(expm1f(dt * a.x), s.x, s.x) + dx * b.x;
        s.y = fmaf(expm1f(dt * a.y), s.y, s.y) + dx * b.y;
        S = pair_of(s.x, s.y);
        y = pair_of(fmaf(s.x, c.x, o.x), fmaf(s.y, c.y, o.y));
    }
    static __device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
};

// VEC (4 or 1) neighbouring values as they lie in memory: fetched ahead of their use without being touched
template <typename T, int VEC> struct RawVec;
template <> struct RawVec<__nv_bfloat16, 4> { using type = uint2; };
template <> struct RawVec<__nv_bfloat16, 1> { using type = __nv_bfloat16; };
template <> struct RawVec<float, 4> { using type = float4; };
template <> struct RawVec<float, 1> { using type = float; };
// (volatile: issued where they stand, ahead of the tokens that run meanwhile)
__device__ __forceinline__ void load_ahead(uint2& r, const void* p) { asm volatile("ld.global.nc.v2.u32 {%0, %1}, [%2];" : "=r"(r.x), "=r"(r.y) : "l"(p)); }
__device__ __forceinline__ void load_ahead(float4& r, const void* p) { asm volatile("ld.global.nc.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(r.x), "=f"(r.y), "=f"(r.z), "=f"(r.w) : "l"(p)); }
__device__ __forceinline__ void load_ahead(float& r, const void* p) { asm volatile("ld.global.nc.f32 %0, [%1];" : "=f"(r) : "l"(p)); }
__device__ __forceinline__ void load_ahead(__nv_bfloat16& r, const void* p) {
    unsigned short u;
    asm volatile("ld.global.nc.u16 %0, [%1];" : "=h"(u) : "l"(p));
    r = __ushort_as_bfloat16(u);
}
template <typename T, int VEC> __device__ __forceinline__ void unpack(float (&v)[VEC], const typename RawVec<T, VEC>::type& r) {
    const T* p = reinterpret_cast<const T*>(&r);
#pragma unroll
    for (int k = 0; k < VEC; k++) v[k] = to_f(p[k]);
}

// grid (channel blocks, portions), 128 threads: L neighbouring lanes share a channel, SPT states each, in registers.  Tokens run in order in chunks of
// TC, whose (dt, dt x) pairs, B and C sit in shared memory; the next chunk's inputs are fetched into registers meanwhile.  Four tokens' parts of y
// at a time are added over the lanes of a channel so that every shuffle halves the tokens a lane still holds.  VX, VB: values per access of the
// rows of x, dt, z (out) and of B, C.
template <typename T, int SPT, int L, int VX, int VB>
__global__ void __launch_bounds__(128, 4) selective_scan_kernel(const SelScan a, T* __restrict__ out) {
    using M = ScanMath<T>;
    constexpr int CH = 128 / L, CP = CH + 8, NP = SPT * L, TC = L <= 2 ? 16 : (NP <= 64 ? 32 : (NP <= 128 ? 16 : 8));
    constexpr int GX = CH / VX, GB = NP / VB;      // accesses per token
    constexpr int E = TC * GX >= 128 ? TC * GX / 128 : 1, EB = TC * GB >= 128 ? TC * GB / 128 : 1;
    static_assert(CH % VX == 0 && NP % VB == 0 && SPT % 4 == 0, "");
    using RX = typename RawVec<T, VX>::type;
    using RB = typename RawVec<T, VB>::type;
    __shared__ float2 dts[TC * CH];
    __shared__ float ys[TC * CP];
    __shared__ __align__(16) float Bs[TC * NP];
    __shared__ __align__(16) float Cs[TC * NP];
    const int tid = threadIdx.x, l = tid % L, ch = tid / L, ch0 = blockIdx.x * CH, s = blockIdx.y, N = a.N, inner = a.inner;
    const int start = a.seqs[s], len = a.seqs[a.seqs_stride + s], rd = a.seqs[2 * a.seqs_stride + s], wr = a.seqs[3 * a.seqs_stride + s];
    const bool live = ch0 + ch < inner;
    const long at = (long)(ch0 + ch) * N + l * SPT;
    float S0[SPT], f0[SPT];
#pragma unroll
    for (int k = 0; k < SPT; k++) S0[k] = f0[k] = 0.f;
    if (live && a.vec_state) {
#pragma unroll
        for (int k = 0; k < SPT; k += 4) {
            if (l * SPT + k < N) {
                const float4 w = load4(a.A + at + k);
                f0[k] = w.x; f0[k + 1] = w.y; f0[k + 2] = w.z; f0[k + 3] = w.w;
                if (rd >= 0) {
                    const float4 u = load4(a.state + (long)rd * a.state_stride + at + k);
                    S0[k] = u.x; S0[k + 1] = u.y; S0[k + 2] = u.z; S0[k + 3] = u.w;
                }
            }
        }
    } else if (live) {
#pragma unroll
        for (int k = 0; k < SPT; k++) {
            if (l * SPT + k < N) {
                f0[k] = a.A[at + k];
                if (rd >= 0) S0[k] = a.state[(long)rd * a.state_stride + at + k];
            }
        }
    }
    // staging: this thread's channels are the same for every token it fetches (GX divides 128)
    const int sc = (tid % GX) * VX;
    const bool sok = ch0 + sc < inner;
    float bias[VX], skip[VX];
#pragma unroll
    for (int k = 0; k < VX; k++) {
        bias[k] = sok ? a.dt_bias[ch0 + sc + k] : 0.f;
        skip[k] = sok ? a.D[ch0 + sc + k] : 0.f;
    }
    const T *xp = (const T*)a.x + (long)start * inner + ch0 + sc, *dp = (const T*)a.dt + (long)start * a.dt_stride + ch0 + sc, *zp = (const T*)a.z + (long)start * a.z_stride + ch0 + sc;
    RX rx[E], rdt[E], rz[E];
    RB rb[EB], rc[EB];
    auto fetch = [&](int t0) {
        const int nt = min(TC, len - t0);
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int tt = (e * 128 + tid) / GX;
            rx[e] = rdt[e] = rz[e] = RX{};
            if (tt < nt && sok) {
                const long t = t0 + tt;
                load_ahead(rx[e], xp + t * inner);
                load_ahead(rdt[e], dp + t * a.dt_stride);
                load_ahead(rz[e], zp + t * a.z_stride);
            }
        }
#pragma unroll
        for (int e = 0; e < EB; e++) {
            const int i = e * 128 + tid, tt = i / GB, n = (i % GB) * VB;
            rb[e] = rc[e] = RB{};
            if (tt < nt && n < N) {
                const long t = start + t0 + tt;
                load_ahead(rb[e], (const T*)a.B + t * a.bc_stride + n);
                load_ahead(rc[e], (const T*)a.C + t * a.bc_stride + n);
            }
        }
    };
    if (len > 0) fetch(0);
    uint64_t S[SPT / 2], f[SPT / 2];
#pragma unroll
    for (int k = 0; k < SPT / 2; k++) {
        S[k] = pair_of(S0[2 * k], S0[2 * k + 1]);
        f[k] = pair_of(M::factor(f0[2 * k]), M::factor(f0[2 * k + 1]));
    }
    for (int t0 = 0; t0 < len; t0 += TC) {
        const int nt = min(TC, len - t0);
        RX cx[E], cz[E];
        __syncthreads();      // the previous chunk is consumed
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = e * 128 + tid, tt = i / GX;
            cx[e] = rx[e];
            cz[e] = rz[e];
            if (i < TC * GX) {
                float x[VX], v[VX];
                unpack<T, VX>(x, rx[e]);
                unpack<T, VX>(v, rdt[e]);
#pragma unroll
                for (int k = 0; k < VX; k++) {
                    const float dt = tt < nt ? M::softplus(v[k] + bias[k]) : 0.f;      // (a padding token leaves the state alone)
                    dts[tt * CH + sc + k] = make_float2(dt, dt * x[k]);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < EB; e++) {
            const int i = e * 128 + tid;
            if (i < TC * GB) {
                float b[VB], c[VB];
                unpack<T, VB>(b, rb[e]);
                unpack<T, VB>(c, rc[e]);
#pragma unroll
                for (int k = 0; k < VB; k++) {
                    const bool in = (i % GB) * VB + k < N;
                    Bs[i * VB + k] = in ? b[k] : 0.f;
                    Cs[i * VB + k] = in ? c[k] : 0.f;
                }
            }
        }
        __syncthreads();
        if (t0 + TC < len) fetch(t0 + TC);
        for (int tg = 0; tg < nt; tg += 4) {
            float y[4];
#pragma unroll
            for (int q = 0; q < 4; q++) {
                const int tt = tg + q;
                const float2 d = dts[tt * CH + ch];
                uint64_t yy = 0;      // (two zeros)
#pragma unroll
                for (int k = 0; k < SPT; k += 4) {
                    const float4 b = load4(Bs + tt * NP + l * SPT + k), c = load4(Cs + tt * NP + l * SPT + k);
                    M::step(S[k / 2], f[k / 2], d.x, d.y, make_float2(b.x, b.y), make_float2(c.x, c.y), yy);
                    M::step(S[k / 2 + 1], f[k / 2 + 1], d.x, d.y, make_float2(b.z, b.w), make_float2(c.z, c.w), yy);
                }
                const float2 two = halves_of(yy);
                y[q] = two.x + two.y;
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
            const int tt = (e * 128 + tid) / GX;
            if (tt < nt && sok) {
                float x[VX], z[VX], o[VX];
                unpack<T, VX>(x, cx[e]);
                unpack<T, VX>(z, cz[e]);
#pragma unroll
                for (int k = 0; k < VX; k++) o[k] = fmaf(skip[k], x[k], ys[tt * CP + sc + k]) * silu_for<T>(z[k]);
                T* to = out + (long)(start + t0 + tt) * inner + ch0 + sc;
                if (VX == 4) store4(to, make_float4(o[0], o[VX > 1 ? 1 : 0], o[VX > 2 ? 2 : 0], o[VX > 3 ? 3 : 0]));
                else to[0] = from_f<T>(o[0]);
            }
        }
    }
    if (wr >= 0 && live) {
        float* w = a.state + (long)wr * a.state_stride + at;
#pragma unroll
        for (int k = 0; k < SPT; k += 4) {
            const float2 p = halves_of(S[k / 2]), q = halves_of(S[k / 2 + 1]);
            const float v[4] = {p.x, p.y, q.x, q.y};
            if (a.vec_state) {
                if (l * SPT + k < N) store4(w + k, make_float4(v[0], v[1], v[2], v[3]));
            } else {
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (l * SPT + k + e < N) w[k + e] = v[e];
            }
        }
    }
}

// One token per portion: grid (blocks of channels x L lanes, portions), no shared memory.  L lanes (a power of two) share a channel, four neighbouring
// states each at a time; what a channel needs besides is read by all of its lanes.
constexpr int kStepThreads = 128;
template <typename T, bool VEC>
__global__ void __launch_bounds__(kStepThreads) selective_scan_step_kernel(const SelScan a, int L, T* __restrict__ out) {
    using M = ScanMath<T>;
    const long i = blockIdx.x * (long)kStepThreads + threadIdx.x;
    const int s = blockIdx.y, N = a.N, l = (int)(i % L), ch = (int)min(i / L, (long)a.inner - 1);      // (lanes behind the last channel repeat it, and store nothing)
    const bool live = i / L < a.inner;
    const long t = a.seqs[s], at = (long)ch * N;
    const int rd = a.seqs[2 * a.seqs_stride + s], wr = a.seqs[3 * a.seqs_stride + s];
    const float x = to_f(((const T*)a.x)[t * a.inner + ch]), z = to_f(((const T*)a.z)[t * a.z_stride + ch]);
    const float dt = M::softplus(to_f(((const T*)a.dt)[t * a.dt_stride + ch]) + a.dt_bias[ch]), dx = dt * x;
    const T *B = (const T*)a.B + t * a.bc_stride, *Cv = (const T*)a.C + t * a.bc_stride;
    const float* Sr = a.state + (long)rd * a.state_stride + at;
    float* Sw = a.state + (long)wr * a.state_stride + at;
    uint64_t y = 0;      // (two zeros)
    for (int n = 4 * l; n < N; n += 4 * L) {
        float4 f, v = make_float4(0.f, 0.f, 0.f, 0.f), b = v, c = v;
        if (VEC) {
            f = load4(a.A + at + n);
            if (rd >= 0) v = load4(Sr + n);
            b = load4(B + n);
            c = load4(Cv + n);
        } else {
            float u[4][4];
#pragma unroll
            for (int k = 0; k < 4; k++) {
                const bool in = n + k < N;
                u[0][k] = in ? a.A[at + n + k] : 0.f;
                u[1][k] = in && rd >= 0 ? Sr[n + k] : 0.f;
                u[2][k] = in ? to_f(B[n + k]) : 0.f;
                u[3][k] = in ? to_f(Cv[n + k]) : 0.f;
            }
            f = make_float4(u[0][0], u[0][1], u[0][2], u[0][3]);
            v = make_float4(u[1][0], u[1][1], u[1][2], u[1][3]);
            b = make_float4(u[2][0], u[2][1], u[2][2], u[2][3]);
            c = make_float4(u[3][0], u[3][1], u[3][2], u[3][3]);
        }
        uint64_t S0 = pair_of(v.x, v.y), S1 = pair_of(v.z, v.w);
        M::step(S0, pair_of(M::factor(f.x), M::factor(f.y)), dt, dx, make_float2(b.x, b.y), make_float2(c.x, c.y), y);
        M::step(S1, pair_of(M::factor(f.z), M::factor(f.w)), dt, dx, make_float2(b.z, b.w), make_float2(c.z, c.w), y);
        if (wr >= 0 && live) {
            const float2 p = halves_of(S0), q = halves_of(S1);
            if (VEC) {
                store4(Sw + n, make_float4(p.x, p.y, q.x, q.y));
            } else {
                const float w[4] = {p.x, p.y, q.x, q.y};
#pragma unroll
                for (int k = 0; k < 4; k++)
                    if (n + k < N) Sw[n + k] = w[k];
            }
        }
    }
    const float2 two = halves_of(y);
    float sum = two.x + two.y;
    for (int o = 1; o < L; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (live && l == 0) out[t * a.inner + ch] = from_f<T>(fmaf(a.D[ch], x, sum) * silu_for<T>(z));
}

}  // namespace ktb

using namespace ktb;

#define SEQ_DISPATCH(dtype, ...)                                                           \
    do {                                                                                   \
        if ((dtype) == KTB200_TYPE_BF16) { using T = __nv_bfloat16; __VA_ARGS__; }         \
        else if ((dtype) == KTB200_TYPE_F32) { using T = float; __VA_ARGS__; }             \
        else { set_error("dtype must be bf16 or f32"); return KTB200_EINVAL; }             \
    } while (0)

extern "C" int ktb200_selective_scan(const ktb200_selective_scan_params* c, void* out, int n_tokens, int dtype, void* stream) {
    if (!c || !c->x || !c->dt_logit || !c->b || !c->c || !c->z || !c->dt_bias || !c->a || !c->d_skip || !c->seqs || !c->state || !out || c->inner <= 0 || c->state_size <= 0 ||
        c->state_size > 256) {
        set_error("selective_scan: bad argument (state size <= 256)");
        return KTB200_EINVAL;
    }
    if (c->n_seqs <= 0 || n_tokens <= 0) return KTB200_OK;
    const int N = c->state_size;
    const size_t esz = dtype == KTB200_TYPE_BF16 ? 2 : 4;
    auto al = [](const void* p, size_t b) { return (reinterpret_cast<uintptr_t>(p) & (b - 1)) == 0; };
    const SelScan a{c->x, c->dt_logit, c->b, c->c, c->z, c->dt_stride, c->bc_stride, c->z_stride, c->dt_bias, c->a, c->d_skip, c->inner, N, c->seqs, c->seqs_stride, c->state,
                    c->state_stride, N % 4 == 0 && c->state_stride % 4 == 0 && al(c->state, 16) && al(c->a, 16)};
    // rows in groups of four where they allow it
    const bool vec = c->inner % 4 == 0 && N % 4 == 0 && c->dt_stride % 4 == 0 && c->z_stride % 4 == 0 && c->bc_stride % 4 == 0 && al(c->x, 4 * esz) && al(c->dt_logit, 4 * esz) &&
                     al(c->z, 4 * esz) && al(c->b, 4 * esz) && al(c->c, 4 * esz) && al(out, 4 * esz);
    const cudaStream_t st = (cudaStream_t)stream;
    if (n_tokens == c->n_seqs) {
        int L = 1;
        while (L < 32 && 4 * L < N) L <<= 1;
        const dim3 grid((unsigned)(((long)c->inner * L + kStepThreads - 1) / kStepThreads), c->n_seqs);
        SEQ_DISPATCH(dtype, {
            if (vec && a.vec_state) selective_scan_step_kernel<T, true><<<grid, kStepThreads, 0, st>>>(a, L, (T*)out);
            else selective_scan_step_kernel<T, false><<<grid, kStepThreads, 0, st>>>(a, L, (T*)out);
        });
        KTB_LAUNCH_CHECK();
        return KTB200_OK;
    }
#define SCAN_LAUNCH(SPT, L)                                                                                     \
    SEQ_DISPATCH(dtype, {                                                                                       \
        const dim3 grid((c->inner + 128 / (L) - 1) / (128 / (L)), c->n_seqs);                                   \
        if (vec) selective_scan_kernel<T, SPT, L, 4, 4><<<grid, 128, 0, st>>>(a, (T*)out);                      \
        else selective_scan_kernel<T, SPT, L, 1, 1><<<grid, 128, 0, st>>>(a, (T*)out);                          \
    })
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
