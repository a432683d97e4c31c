// Mamba-2 (state-space duality): a recurrent mixer whose matrix state per head decays by one number per token and head
// (libktb200_seq.so).
//
//   ktb200_conv_silu  causal filter of `taps` taps along time with bias on a run of channels, then SiLU, over prompt portions and decode steps alike
//   ktb200_ssd_conv   prompt portions: causal filter of `taps` taps along time with bias on the [x | B | C] channels, then SiLU; the last taps - 1
//                     inputs of every portion go to its state row
//   ktb200_ssd_scan   per portion and head p (group j = p / (P / J)), tokens in order, fp32:
//                         dt = softplus(. + dt_bias_p), S <- exp(-exp(A_log_p) dt) S + dt B_j x_p^T, y = S^T C_j + D_p x_p
//                     token by token on CUDA cores, or (bf16) in chunks of 64 tokens on the tensor cores
//   ktb200_ssd_step   decode steps (one token per portion): the filter, SiLU and the recurrence in one launch
//   ktb200_gated_group_norm   y silu(z), every one of `groups` equal parts to unit rms, times a weight and a constant
//
// State row of a sequence and layer (fp32): [ S heads x state x vdim | filter inputs (taps - 1) x channels, oldest first ], read from the row
// seqs[2][s] (or zeros when -1) and written to the row seqs[3][s]: the caller double-buffers the rows.  Storage type T (bf16 or float) for
// projections, filter weights and the filtered channels; steps, decays, the state and everything read from it are fp32.
#include <cuda_bf16.h>

#include "common.cuh"
#include "seq_common.cuh"
#include "mma_tile.cuh"

namespace ktb {

__device__ __forceinline__ float ssd_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// ------------------------------------------------------------------------------------------------ filter + SiLU over prompt portions
// grid (token blocks, channel blocks); a thread owns VEC consecutive channels and runs over `tile` tokens (kConvTokens; 1 when every portion is one token) with the last TAPS - 1 inputs
// in registers (TAPS = 0: any number of taps, one channel, inputs read again per token).
constexpr int kConvTokens = 16, kConvThreads = 128, kConvAhead = 4;
template <typename T, int VEC> __device__ __forceinline__ void load_vec(float (&v)[VEC], const T* p) {
    if (VEC == 4) {
        const float4 u = load4(p);
        v[0] = u.x; v[VEC > 1 ? 1 : 0] = u.y; v[VEC > 2 ? 2 : 0] = u.z; v[VEC > 3 ? 3 : 0] = u.w;
    } else {
        v[0] = to_f(p[0]);
    }
}
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kConvThreads) conv_silu_kernel(const T* __restrict__ in, long stride, const T* __restrict__ w, const T* __restrict__ bias, int taps_rt, int C,
                                                                const int* __restrict__ seq_of, const int* __restrict__ seqs, int seqs_stride, float* __restrict__ state,
                                                                long state_stride, long conv_off, T* __restrict__ out, int n_tokens, int tile) {
    const int c = (blockIdx.y * kConvThreads + threadIdx.x) * VEC;
    if (c >= C) return;
    const int t0 = blockIdx.x * tile, t1 = min(n_tokens, t0 + tile);
    constexpr int BACK = TAPS > 1 ? TAPS - 1 : 1;
    float win[BACK][VEC], wv[TAPS > 0 ? TAPS : 1][VEC], bv[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) {
        bv[e] = bias ? to_f(bias[c + e]) : 0.f;
        if (TAPS > 0)
#pragma unroll
            for (int j = 0; j < TAPS; j++) wv[j][e] = to_f(w[(long)(c + e) * TAPS + j]);
    }
    int cur = -1, start = 0, len = 0, rd = -1, wr = -1;
    for (int tb = t0; tb < t1; tb += kConvAhead) {
        float in_rows[kConvAhead][VEC];      // the next tokens' inputs, asked for together
        if (TAPS > 0) {
#pragma unroll
            for (int q = 0; q < kConvAhead; q++)
                if (tb + q < t1) load_vec<T, VEC>(in_rows[q], in + (long)(tb + q) * stride + c);
        }
#pragma unroll
        for (int q = 0; q < kConvAhead; q++) {
            const int t = tb + q;
            if (t >= t1) break;
            const int s = seq_of[t];
            const bool fresh = s != cur;      // another portion, or this thread's first token: fetch the inputs ahead of it
            if (fresh) {
                cur = s;
                start = seqs[s]; len = seqs[seqs_stride + s]; rd = seqs[2 * seqs_stride + s]; wr = seqs[3 * seqs_stride + s];
            }
            const int off = t - start;
            const ConvRows<T> cv{in + (long)start * stride, stride, w, TAPS > 0 ? TAPS : taps_rt, C, rd >= 0 ? state + (long)rd * state_stride + conv_off : nullptr,
                                 wr >= 0 ? state + (long)wr * state_stride + conv_off : nullptr, off};
            if (TAPS == 0) {
                out[(long)t * C + c] = from_f<T>(silu_for<T>(cv.value(c, c) + bv[0]));
                if (off == len - 1 && wr >= 0) cv.store_tail(c, c);
                continue;
            }
            if (fresh && TAPS > 1) {
#pragma unroll
                for (int j = 0; j < TAPS - 1; j++)
#pragma unroll
                    for (int e = 0; e < VEC; e++) win[j][e] = cv.input(off - (TAPS - 1) + j, c + e, c + e);
            }
            float y[VEC];
#pragma unroll
            for (int e = 0; e < VEC; e++) {
                float a = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS - 1; j++) a = fmaf(wv[j][e], win[j][e], a);
                y[e] = silu_for<T>(fmaf(wv[TAPS - 1 > 0 ? TAPS - 1 : 0][e], in_rows[q][e], a) + bv[e]);
#pragma unroll
                for (int j = 0; j + 1 < TAPS - 1; j++) win[j][e] = win[j + 1][e];
                if (TAPS > 1) win[BACK - 1][e] = in_rows[q][e];
            }
            if (VEC == 4) store4(out + (long)t * C + c, make_float4(y[0], y[VEC > 1 ? 1 : 0], y[VEC > 2 ? 2 : 0], y[VEC > 3 ? 3 : 0]));
            else out[(long)t * C + c] = from_f<T>(y[0]);
            if (TAPS > 1 && off == len - 1 && wr >= 0) {
#pragma unroll
                for (int j = 0; j < TAPS - 1; j++)
#pragma unroll
                    for (int e = 0; e < VEC; e++) cv.after[(long)j * C + c + e] = win[j][e];
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ the recurrence over prompt portions
// grid (portions, heads, column blocks of 32 value columns); 8 warps; thread (warp w, lane) keeps S[n][col] for a contiguous run of state
// rows n in registers.  Tokens run in order in chunks of kSsdChunk staged in shared memory, the next chunk's inputs fetched into registers
// while the current one runs; per token every warp leaves its part of y in shared memory, summed in warp order once per chunk.
constexpr int kSsdChunk = 16, kSsdWarps = 8, kSsdRows = 32;      // state size <= 256
template <typename T, int ROWS>
__global__ void __launch_bounds__(256, 2) ssd_scan_kernel(const T* __restrict__ xbc, const T* __restrict__ dt_in, long dt_stride, const float* __restrict__ dt_bias,
                                                          const float* __restrict__ a_log, const float* __restrict__ Dv, int P, int J, int N, int dv, const int* __restrict__ seqs,
                                                          int seqs_stride, float* __restrict__ state, long state_stride, float* __restrict__ y_out) {
    extern __shared__ __align__(16) float sm[];
    const int rpt = (((N + kSsdWarps - 1) / kSsdWarps) + 3) & ~3, np = rpt * kSsdWarps;
    float* Bs = sm;                              // [chunk][np]
    float* Cs = Bs + kSsdChunk * np;             // [chunk][np]
    float* xs = Cs + kSsdChunk * np;             // [chunk][32]
    float* sc = xs + kSsdChunk * 32;             // [chunk][2]: decay, dt
    float* part = sc + kSsdChunk * 2;            // [chunk][warps][32]
    const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * 32, j = h / (P / J), inner = P * dv, C = inner + 2 * J * N;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, col = c0 + lane;
    const int start = seqs[s], len = seqs[seqs_stride + s], rd = seqs[2 * seqs_stride + s], wr = seqs[3 * seqs_stride + s];
    float S[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; r++) {
        const int n = warp * rpt + r;
        S[r] = (rd >= 0 && r < rpt && n < N && col < dv) ? state[(long)rd * state_stride + ((long)h * N + n) * dv + col] : 0.f;
    }
    const float rate = expf(a_log[h]), bias = dt_bias[h], Dh = Dv[h];
    constexpr int E = kSsdChunk * ROWS * kSsdWarps / 256;      // staged state-row values per thread and array, at most
    float rb[E], rc[E], rx[2], rdt = 0.f;
    auto fetch = [&](int t0) {
        const int nt = min(kSsdChunk, len - t0);
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = threadIdx.x + e * 256;
            rb[e] = rc[e] = 0.f;
            if (i < nt * np) {
                const int tt = i / np, n = i - tt * np;
                if (n < N) {
                    const T* row = xbc + (long)(start + t0 + tt) * C + inner + j * N + n;
                    rb[e] = to_f(row[0]);
                    rc[e] = to_f(row[J * N]);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int i = threadIdx.x + e * 256, c = c0 + (i & 31);
            rx[e] = (i < nt * 32 && c < dv) ? to_f(xbc[(long)(start + t0 + (i >> 5)) * C + h * dv + c]) : 0.f;
        }
        if (threadIdx.x < nt) rdt = to_f(dt_in[(long)(start + t0 + threadIdx.x) * dt_stride + h]);
    };
    if (len > 0) fetch(0);
    for (int t0 = 0; t0 < len; t0 += kSsdChunk) {
        const int nt = min(kSsdChunk, len - t0);
        __syncthreads();      // the previous chunk is consumed
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = threadIdx.x + e * 256;
            if (i < nt * np) { Bs[i] = rb[e]; Cs[i] = rc[e]; }
        }
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int i = threadIdx.x + e * 256;
            if (i < nt * 32) xs[i] = rx[e];
        }
        if (threadIdx.x < nt) {
            const float dt = ssd_softplus(rdt + bias);
            sc[2 * threadIdx.x] = expf(-rate * dt);
            sc[2 * threadIdx.x + 1] = dt;
        }
        __syncthreads();
        if (t0 + kSsdChunk < len) fetch(t0 + kSsdChunk);
#pragma unroll 2
        for (int tt = 0; tt < nt; tt++) {
            const float a = sc[2 * tt], xd = xs[tt * 32 + lane] * sc[2 * tt + 1];
            const float4* br = reinterpret_cast<const float4*>(Bs + tt * np + warp * rpt);
            const float4* cr = reinterpret_cast<const float4*>(Cs + tt * np + warp * rpt);
            float y0 = 0.f, y1 = 0.f;
#pragma unroll
            for (int r4 = 0; r4 < ROWS / 4; r4++) {
                if (4 * r4 < rpt) {
                    const float4 b = br[r4], c = cr[r4];
                    S[4 * r4] = fmaf(a, S[4 * r4], b.x * xd);
                    y0 = fmaf(S[4 * r4], c.x, y0);
                    S[4 * r4 + 1] = fmaf(a, S[4 * r4 + 1], b.y * xd);
                    y1 = fmaf(S[4 * r4 + 1], c.y, y1);
                    S[4 * r4 + 2] = fmaf(a, S[4 * r4 + 2], b.z * xd);
                    y0 = fmaf(S[4 * r4 + 2], c.z, y0);
                    S[4 * r4 + 3] = fmaf(a, S[4 * r4 + 3], b.w * xd);
                    y1 = fmaf(S[4 * r4 + 3], c.w, y1);
                }
            }
            part[(tt * kSsdWarps + warp) * 32 + lane] = y0 + y1;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nt * 32; i += blockDim.x) {
            const int tt = i >> 5, c = c0 + (i & 31);
            float y = 0.f;
#pragma unroll
            for (int w = 0; w < kSsdWarps; w++) y += part[(tt * kSsdWarps + w) * 32 + (i & 31)];
            if (c < dv) y_out[(long)(start + t0 + tt) * inner + h * dv + c] = fmaf(Dh, xs[i], y);
        }
    }
    if (wr >= 0) {
#pragma unroll
        for (int r = 0; r < ROWS; r++) {
            const int n = warp * rpt + r;
            if (r < rpt && n < N && col < dv) state[(long)wr * state_stride + ((long)h * N + n) * dv + col] = S[r];
        }
    }
}

// ------------------------------------------------------------------------------------------------ the recurrence, chunked, tensor cores (bf16)
// grid (portions, heads, column blocks of 32 value columns), 8 warps.  Tokens run in chunks of 64 with L the running sum of log decays inside
// the chunk (fp32, L <= 0 and falling, so every factor below is at most one):
//     y_i = exp(L_i) C_i S + sum_{j <= i} (C_i . B_j) exp(L_i - L_j) dt_j x_j + D x_i          S <- exp(L_last) S + sum_j B_j (exp(L_last - L_j) dt_j x_j)^T
// as m16n8k16 bf16 MMAs with fp32 accumulators.  B, C and x are bf16 as they come; what the fp32 factors touch — the weighted scores, the weighted
// x rows and S as an operand — enters as the sum of two bf16 terms (about 16 bits of mantissa).  Warps 0..3 make the outputs of 16 tokens each;
// warps 4..7 meanwhile take the chunk into S, whose fp32 accumulators they keep from chunk to chunk (MT tiles of 16 state rows each), and
// publish it for the next chunk once the output warps have read the old one.  The next chunk's rows are on their way in the other stage.
constexpr int kChunkQ = 64, kChunkCols = 32, kChunkLd = kChunkCols + 8;
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
static size_t ssd_chunk_smem(int N) { return ((size_t)4 * kChunkQ * (N + 8) + 4 * kChunkQ * kChunkLd + (size_t)2 * N * kChunkLd) * 2 + 8 * kChunkQ * sizeof(float); }

// The outputs of the chunk's tokens 16 W .. 16 W + 15 by one warp: C S and the scores against the chunk's tokens up to its own in one pass over
// the state rows, then the weighted scores times x.  W is a template parameter so that the tiles above the diagonal fall away at compile time
// and the operand loads of a step are all issued ahead of its MMAs.
template <int W>
__device__ __forceinline__ void ssd_chunk_outputs(const __nv_bfloat16* Cs, const __nv_bfloat16* Bs, const __nv_bfloat16* Xs, const __nv_bfloat16* Sh, const float* Ls, const float* eL,
                                                  const float* dts, int N, int nt, bool more, float Dh, float* __restrict__ y, long inner, int cols) {
    constexpr int LD = kChunkLd;
    const int ldn = N + 8, n16 = N >> 4, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3;
    float Y[4][4], G[2 * W + 2][4];
#pragma unroll
    for (int n = 0; n < 4; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) Y[n][e] = 0.f;
#pragma unroll
    for (int n = 0; n < 2 * W + 2; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) G[n][e] = 0.f;
    const __nv_bfloat16* ca = Cs + (W * 16 + (lane & 15)) * ldn + 8 * (lane >> 4);
    const __nv_bfloat16* ba = Bs + ((lane & 7) + 8 * (lane >> 4)) * ldn + 8 * ((lane >> 3) & 1);
    const __nv_bfloat16* sa = Sh + (lane & 15) * LD + 8 * (lane >> 4);
#pragma unroll 2
    for (int kk = 0; kk < n16; kk++) {
        uint32_t a[4], b[W + 1][4], st[2][2][4];
        ldmatrix_x4(a, ca + kk * 16);
#pragma unroll
        for (int np = 0; np <= W; np++) ldmatrix_x4(b[np], ba + np * 16 * ldn + kk * 16);
#pragma unroll
        for (int term = 0; term < 2; term++)
#pragma unroll
            for (int vp = 0; vp < 2; vp++) ldmatrix_x4_trans(st[term][vp], sa + (term * N + kk * 16) * LD + vp * 16);
#pragma unroll
        for (int np = 0; np <= W; np++) {
            mma_bf16_16816(G[2 * np], a, b[np][0], b[np][1]);
            mma_bf16_16816(G[2 * np + 1], a, b[np][2], b[np][3]);
        }
#pragma unroll
        for (int term = 0; term < 2; term++)
#pragma unroll
            for (int vp = 0; vp < 2; vp++) {
                mma_bf16_16816(Y[2 * vp], a, st[term][vp][0], st[term][vp][1]);
                mma_bf16_16816(Y[2 * vp + 1], a, st[term][vp][2], st[term][vp][3]);
            }
    }
    if (more) asm volatile("bar.arrive 2, 256;" ::: "memory");      // the old state is read
    const int iA = W * 16 + gq, iB = iA + 8;
    const float LA = Ls[iA], LB = Ls[iB], eA = eL[iA], eB = eL[iB];
#pragma unroll
    for (int n = 0; n < 4; n++) {
        Y[n][0] *= eA;
        Y[n][1] *= eA;
        Y[n][2] *= eB;
        Y[n][3] *= eB;
    }
#pragma unroll
    for (int kk = 0; kk <= W; kk++) {
        uint32_t b[2][4];
#pragma unroll
        for (int vp = 0; vp < 2; vp++) ldmatrix_x4_trans(b[vp], Xs + (kk * 16 + (lane & 15)) * LD + vp * 16 + 8 * (lane >> 4));
#pragma unroll
        for (int n = 2 * kk; n < 2 * kk + 2; n++) {
            const int jj = n * 8 + 2 * tq;
            const float2 Lj = *reinterpret_cast<const float2*>(Ls + jj), dj = *reinterpret_cast<const float2*>(dts + jj);
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const float f = __expf((e < 2 ? LA : LB) - ((e & 1) ? Lj.y : Lj.x)) * ((e & 1) ? dj.y : dj.x);
                G[n][e] = kk < W || jj + (e & 1) <= (e < 2 ? iA : iB) ? G[n][e] * f : 0.f;      // (only the diagonal tile has anything to mask)
            }
        }
        uint32_t hi[4], lo[4];
        split_bf16(G[2 * kk][0], G[2 * kk][1], hi[0], lo[0]);
        split_bf16(G[2 * kk][2], G[2 * kk][3], hi[1], lo[1]);
        split_bf16(G[2 * kk + 1][0], G[2 * kk + 1][1], hi[2], lo[2]);
        split_bf16(G[2 * kk + 1][2], G[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int vp = 0; vp < 2; vp++) {
            mma_bf16_16816(Y[2 * vp], hi, b[vp][0], b[vp][1]);
            mma_bf16_16816(Y[2 * vp + 1], hi, b[vp][2], b[vp][3]);
        }
#pragma unroll
        for (int vp = 0; vp < 2; vp++) {
            mma_bf16_16816(Y[2 * vp], lo, b[vp][0], b[vp][1]);
            mma_bf16_16816(Y[2 * vp + 1], lo, b[vp][2], b[vp][3]);
        }
    }
#pragma unroll
    for (int n = 0; n < 4; n++) {
        const int c = n * 8 + 2 * tq;
        if (c < cols) {
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int i = e ? iB : iA;
                if (i < nt) {
                    const uint32_t u = *reinterpret_cast<const uint32_t*>(Xs + i * LD + c);
                    *reinterpret_cast<float2*>(y + i * inner + c) = make_float2(fmaf(Dh, __uint_as_float(u << 16), Y[n][e]), fmaf(Dh, __uint_as_float(u & 0xffff0000u), Y[n][e + 1]));
                }
            }
        }
    }
}

template <int MT>
__global__ void __launch_bounds__(256, MT <= 2 ? 2 : 1) ssd_chunk_kernel(const __nv_bfloat16* __restrict__ xbc, const __nv_bfloat16* __restrict__ dt_in, long dt_stride,
                                                                         const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ Dv, int P, int J, int N,
                                                                         int dv, const int* __restrict__ seqs, int seqs_stride, float* __restrict__ state, long state_stride,
                                                                         float* __restrict__ y_out) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    constexpr int Q = kChunkQ, LD = kChunkLd;
    const int ldn = N + 8;
    __nv_bfloat16* const ring = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // two stages of C [Q][ldn] | B [Q][ldn] | x [Q][LD]
    const int stage_elems = 2 * Q * ldn + Q * LD;
    __nv_bfloat16* Xh = ring + 2 * stage_elems;                          // [2][Q][LD]: the weighted rows, two terms
    __nv_bfloat16* Sh = Xh + 2 * Q * LD;                                 // [2][N][LD]: the state, two terms
    float* const factors = reinterpret_cast<float*>(Sh + 2 * N * LD);    // two sets of L, exp(L), dt, exp(L_last - L) dt, [Q] each
    const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kChunkCols, j = h / (P / J), inner = P * dv, C = inner + 2 * J * N;
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, warp = wid & 3, gq = lane >> 2, tq = lane & 3;
    const int start = seqs[s], len = seqs[seqs_stride + s], rd = seqs[2 * seqs_stride + s], wr = seqs[3 * seqs_stride + s];
    const bool reads_out = wid < 4;      // warps 0..3 make the outputs, warps 4..7 carry the state
    const float rate = expf(a_log[h]), bias = dt_bias[h], Dh = Dv[h];
    float S[MT][4][4];      // state warps: [tile of 16 state rows][8 columns]
    if (!reads_out) {
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int n = 0; n < 4; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int r = (warp * MT + m) * 16 + gq + 8 * (e >> 1), c = c0 + n * 8 + 2 * tq + (e & 1);
                    S[m][n][e] = rd >= 0 && r < N && c < dv ? state[(long)rd * state_stride + ((long)h * N + r) * dv + c] : 0.f;
                }
    }
    auto publish = [&]() {      // S as two bf16 terms for the next chunk
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int n = 0; n < 4; n++)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int r = (warp * MT + m) * 16 + gq + 4 * e;
                    uint32_t hi, lo;
                    split_bf16(S[m][n][e], S[m][n][e + 1], hi, lo);
                    if (r < N) {
                        *reinterpret_cast<uint32_t*>(Sh + r * LD + n * 8 + 2 * tq) = hi;
                        *reinterpret_cast<uint32_t*>(Sh + (N + r) * LD + n * 8 + 2 * tq) = lo;
                    }
                }
    };
    if (!reads_out) publish();
    const int nc = N >> 3;      // 16-byte pieces per B or C row
    auto fetch = [&](int t0, int stage) {
        const int nt = min(Q, len - t0);
        __nv_bfloat16 *Cd = ring + stage * stage_elems, *Bd = Cd + Q * ldn, *Xd = Bd + Q * ldn;
        for (int i = tid; i < Q * nc; i += 256) {
            const int r = i / nc, c = i - r * nc;
            const __nv_bfloat16* src = xbc + (long)(start + t0 + (r < nt ? r : 0)) * C + inner + j * N + c * 8;
            cp_async16(Bd + r * ldn + c * 8, src, r < nt);
            cp_async16(Cd + r * ldn + c * 8, src + J * N, r < nt);
        }
        for (int i = tid; i < Q * (kChunkCols / 8); i += 256) {
            const int r = i >> 2, c = (i & 3) * 8;
            const bool ok = r < nt && c0 + c < dv;
            cp_async16(Xd + r * LD + c, ok ? xbc + (long)(start + t0 + r) * C + h * dv + c0 + c : xbc, ok);
        }
    };
    // the factors of the chunk at t0 by one warp, tokens 2 lane and 2 lane + 1 per lane; the step logits are asked for ahead of time
    float dt_next[2];
    auto fetch_dt = [&](int t0) {
#pragma unroll
        for (int e = 0; e < 2; e++) dt_next[e] = t0 + 2 * lane + e < len ? __bfloat162float(dt_in[(long)(start + t0 + 2 * lane + e) * dt_stride + h]) : 0.f;
    };
    auto make_factors = [&](int t0, int set) {
        float *Ls = factors + set * 4 * Q, *eL = Ls + Q, *dts = eL + Q, *wts = dts + Q;
        float dt[2], la[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
            dt[e] = t0 + 2 * lane + e < len ? ssd_softplus(dt_next[e] + bias) : 0.f;
            la[e] = -rate * dt[e];
        }
        float run = la[0] + la[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += up;
        }
        const float last = __shfl_sync(0xffffffffu, run, 31);
        const float L0 = run - la[1];
        Ls[2 * lane] = L0;
        Ls[2 * lane + 1] = run;
        eL[2 * lane] = expf(L0);
        eL[2 * lane + 1] = expf(run);
        dts[2 * lane] = dt[0];
        dts[2 * lane + 1] = dt[1];
        wts[2 * lane] = expf(last - L0) * dt[0];
        wts[2 * lane + 1] = expf(last - run) * dt[1];
    };
    const int factor_warp = 7;
    if (len > 0) {
        fetch(0, 0);
        if (wid == factor_warp) {
            fetch_dt(0);
            make_factors(0, 0);
        }
    }
    int stage = 0;
    for (int t0 = 0; t0 < len; t0 += Q, stage ^= 1) {
        const int nt = min(Q, len - t0);
        const __nv_bfloat16 *Cs = ring + stage * stage_elems, *Bs = Cs + Q * ldn, *Xs = Bs + Q * ldn;
        const float *Ls = factors + stage * 4 * Q, *eL = Ls + Q, *dts = eL + Q, *wts = dts + Q;
        cp_async_wait_all();
        __syncthreads();      // this chunk, its factors and the state ahead of it are there; the other stage is free
        if (t0 + Q < len) {
            fetch(t0 + Q, stage ^ 1);
            if (wid == factor_warp) fetch_dt(t0 + Q);
        }
        if (!reads_out) {
            for (int i = tid - 128; i < Q * kChunkCols / 2; i += 128) {      // the weighted x rows
                const int r = i / (kChunkCols / 2), c = (i % (kChunkCols / 2)) * 2;
                const uint32_t u = *reinterpret_cast<const uint32_t*>(Xs + r * LD + c);
                uint32_t hi, lo;
                split_bf16(__uint_as_float(u << 16) * wts[r], __uint_as_float(u & 0xffff0000u) * wts[r], hi, lo);
                *reinterpret_cast<uint32_t*>(Xh + r * LD + c) = hi;
                *reinterpret_cast<uint32_t*>(Xh + (Q + r) * LD + c) = lo;
            }
            asm volatile("bar.sync 1, 128;" ::: "memory");      // among the state warps
            const float keep = eL[Q - 1];
            const int k16 = (nt + 15) >> 4;
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int n = 0; n < 4; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) S[m][n][e] *= keep;
            if (warp * MT * 16 < N) {
#pragma unroll 2
                for (int kk = 0; kk < k16; kk++) {
                    uint32_t x[2][2][4];
#pragma unroll
                    for (int term = 0; term < 2; term++)
#pragma unroll
                        for (int vp = 0; vp < 2; vp++) ldmatrix_x4_trans(x[term][vp], Xh + (term * Q + kk * 16 + (lane & 15)) * LD + vp * 16 + 8 * (lane >> 4));
#pragma unroll
                    for (int m = 0; m < MT; m++) {
                        const int r0 = (warp * MT + m) * 16;
                        if (r0 < N) {
                            uint32_t a[4];
                            ldmatrix_x4_trans(a, Bs + (kk * 16 + (lane & 7) + 8 * (lane >> 4)) * ldn + r0 + 8 * ((lane >> 3) & 1));
#pragma unroll
                            for (int term = 0; term < 2; term++)
#pragma unroll
                                for (int vp = 0; vp < 2; vp++) {
                                    mma_bf16_16816(S[m][2 * vp], a, x[term][vp][0], x[term][vp][1]);
                                    mma_bf16_16816(S[m][2 * vp + 1], a, x[term][vp][2], x[term][vp][3]);
                                }
                        }
                    }
                }
            }
            if (t0 + Q < len) {
                if (wid == factor_warp) make_factors(t0 + Q, stage ^ 1);
                asm volatile("bar.sync 2, 256;" ::: "memory");      // the output warps have read the old state
                publish();
            }
            continue;
        }
        if (warp * 16 < nt) {
            float* y = y_out + (long)(start + t0) * inner + h * dv + c0;
            const bool more = t0 + Q < len;
            if (warp == 0) ssd_chunk_outputs<0>(Cs, Bs, Xs, Sh, Ls, eL, dts, N, nt, more, Dh, y, inner, dv - c0);
            else if (warp == 1) ssd_chunk_outputs<1>(Cs, Bs, Xs, Sh, Ls, eL, dts, N, nt, more, Dh, y, inner, dv - c0);
            else if (warp == 2) ssd_chunk_outputs<2>(Cs, Bs, Xs, Sh, Ls, eL, dts, N, nt, more, Dh, y, inner, dv - c0);
            else ssd_chunk_outputs<3>(Cs, Bs, Xs, Sh, Ls, eL, dts, N, nt, more, Dh, y, inner, dv - c0);
        }
    }
    if (!reads_out && wr >= 0) {
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int n = 0; n < 4; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int r = (warp * MT + m) * 16 + gq + 8 * (e >> 1), c = c0 + n * 8 + 2 * tq + (e & 1);
                    if (r < N && c < dv) state[(long)wr * state_stride + ((long)h * N + r) * dv + c] = S[m][n][e];
                }
    }
}

// ------------------------------------------------------------------------------------------------ one token per portion
// grid (portions, heads, column blocks of `cpb` columns); a thread owns VEC columns of every `rows_par`-th state row, kStepRows of which it
// requests before the filter of this head's x columns and its group's B and C runs.  The group's first head keeps the filter inputs of B and C.
constexpr int kStepRows = 8;
template <typename T, int VEC>
__global__ void __launch_bounds__(256) ssd_step_kernel(const T* __restrict__ proj, long stride, int xbc_off, int dt_off, const T* __restrict__ w, const T* __restrict__ bias, int taps,
                                                       const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ Dv, int P, int J, int N, int dv,
                                                       const int* __restrict__ seqs, int seqs_stride, float* __restrict__ state, long state_stride, long conv_off,
                                                       float* __restrict__ y_out, int cpb) {
    extern __shared__ __align__(16) float sm[];
    const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * cpb, ncol = min(cpb, dv - c0), j = h / (P / J), inner = P * dv, C = inner + 2 * J * N;
    const int t = seqs[s], rd = seqs[2 * seqs_stride + s], wr = seqs[3 * seqs_stride + s];
    float* xs = sm;                         // [cpb]
    float* Bs = xs + cpb;                   // [N]
    float* Cs = Bs + N;                     // [N]
    float* red = Cs + N;                    // [rows_par][cpb]
    const int tcol = cpb / VEC, rows_par = blockDim.x / tcol;      // (cpb <= 256, a multiple of VEC)
    const int tc = threadIdx.x % tcol, tr = threadIdx.x / tcol, cc = tc * VEC;
    const bool mine = tr < rows_par && cc < ncol;
    const float* Sr = state + (long)rd * state_stride + (long)h * N * dv + c0 + cc;
    float* Sw = state + (long)wr * state_stride + (long)h * N * dv + c0 + cc;
    float v[kStepRows][VEC];
    auto request = [&](int base) {
#pragma unroll
        for (int k = 0; k < kStepRows; k++) {
            const int n = base + k * rows_par + tr;
            if (mine && rd >= 0 && n < N) {
                load_vec<float, VEC>(v[k], Sr + (long)n * dv);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; e++) v[k][e] = 0.f;
            }
        }
    };
    request(0);
    const ConvRows<T> cv{proj + (long)t * stride + xbc_off, stride, w, taps, C, rd >= 0 ? state + (long)rd * state_stride + conv_off : nullptr,
                         wr >= 0 ? state + (long)wr * state_stride + conv_off : nullptr, 0};
    const bool keeps_bc = h % (P / J) == 0 && blockIdx.z == 0;
    for (int i = threadIdx.x; i < ncol + 2 * N; i += blockDim.x) {
        const bool is_x = i < ncol;
        const int c = is_x ? h * dv + c0 + i : inner + (i - ncol < N ? j * N + i - ncol : J * N + j * N + i - ncol - N);
        const float y = act_silu(cv.value(c, c) + to_f(bias[c]));
        if (is_x) xs[i] = y;
        else Bs[i - ncol] = y;      // (Cs follows Bs)
        if (wr >= 0 && (is_x || keeps_bc)) cv.store_tail(c, c);
    }
    const float dt = ssd_softplus(to_f(proj[(long)t * stride + dt_off + h]) + dt_bias[h]);
    const float a = expf(-expf(a_log[h]) * dt);
    __syncthreads();
    float xd[VEC], y[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) {
        xd[e] = mine ? xs[cc + e] * dt : 0.f;
        y[e] = 0.f;
    }
    for (int base = 0; base < N; base += kStepRows * rows_par) {
        if (base) request(base);
#pragma unroll
        for (int k = 0; k < kStepRows; k++) {
            const int n = base + k * rows_par + tr;
            if (mine && n < N) {
                const float b = Bs[n], c = Cs[n];
#pragma unroll
                for (int e = 0; e < VEC; e++) {
                    v[k][e] = fmaf(a, v[k][e], b * xd[e]);
                    y[e] = fmaf(v[k][e], c, y[e]);
                }
                if (wr >= 0) {
                    if (VEC == 4) store4(Sw + (long)n * dv, make_float4(v[k][0], v[k][VEC > 1 ? 1 : 0], v[k][VEC > 2 ? 2 : 0], v[k][VEC > 3 ? 3 : 0]));
                    else Sw[(long)n * dv] = v[k][0];
                }
            }
        }
    }
    if (mine) {
#pragma unroll
        for (int e = 0; e < VEC; e++) red[tr * cpb + cc + e] = y[e];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < ncol; i += blockDim.x) {
        float o = 0.f;
        for (int r = 0; r < rows_par; r++) o += red[r * cpb + i];
        y_out[(long)t * inner + h * dv + c0 + i] = fmaf(Dv[h], xs[i], o);
    }
}

// ------------------------------------------------------------------------------------------------ gate, then grouped norm
// grid (tokens, groups): u = y silu(z) of one part in shared memory, its mean square, out = u inv w out_scale into rows of any stride
template <typename T>
__global__ void __launch_bounds__(512) gated_group_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, long z_stride, const T* __restrict__ w, float eps, float out_scale,
                                                               T* __restrict__ out, long out_stride, int n, int vec) {
    extern __shared__ __align__(16) float u[];
    __shared__ float red[32];
    const long t = blockIdx.x;
    const int lo = blockIdx.y * n;
    const float* yr = y + t * (long)gridDim.y * n + lo;
    const T* zr = z + t * z_stride + lo;
    const T* wr = w + lo;
    T* o = out + t * out_stride + lo;
    float s = 0.f;
    if (vec) {
        for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
            const float4 a = load4(yr + i), g = load4(zr + i);
            const float4 v = make_float4(a.x * act_silu(g.x), a.y * act_silu(g.y), a.z * act_silu(g.z), a.w * act_silu(g.w));
            store4(u + i, v);
            s += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
        const float inv = out_scale / sqrtf(block_sum(s, red) / (float)n + eps);
        for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
            const float4 v = load4(u + i), g = load4(wr + i);
            store4(o + i, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
        }
        return;
    }
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = yr[i] * act_silu(to_f(zr[i]));
        u[i] = v;
        s += v * v;
    }
    const float inv = out_scale / sqrtf(block_sum(s, red) / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += blockDim.x) o[i] = from_f<T>(u[i] * inv * to_f(wr[i]));
}

}  // namespace ktb

using namespace ktb;

#define SEQ_DISPATCH(dtype, ...)                                                           \
    do {                                                                                   \
        if ((dtype) == KTB200_TYPE_BF16) { using T = __nv_bfloat16; __VA_ARGS__; }         \
        else if ((dtype) == KTB200_TYPE_F32) { using T = float; __VA_ARGS__; }             \
        else { set_error("dtype must be bf16 or f32"); return KTB200_EINVAL; }             \
    } while (0)
#define GRANT_SMEM(kernel, smem)                                                                                                       \
    do {                                                                                                                               \
        static size_t granted = 46 * 1024; /* less the kernels' static shared memory */                                               \
        if ((smem) > granted) { KTB_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem))); granted = (smem); } \
    } while (0)

static bool ssd_aligned(const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }
static bool ssd_bad(const ktb200_ssd_params* c) {
    return !c || !c->proj || !c->conv_w || !c->conv_b || !c->dt_bias || !c->a_log || !c->d_skip || !c->seqs || !c->state || c->heads <= 0 || c->groups <= 0 || c->heads % c->groups ||
           c->state_size <= 0 || c->vdim <= 0 || c->taps < 1;
}

extern "C" int ktb200_conv_silu(const void* in, long in_stride, const void* conv_w, const void* conv_b, int taps, int channels, const int* seq_of, const int* seqs, int seqs_stride,
                                float* state, long state_stride, long conv_off, void* out, int n_tokens, int n_seqs, int dtype, void* stream) {
    if (!in || !conv_w || !out || !seq_of || !seqs || taps < 1 || (taps > 1 && !state) || channels <= 0) { set_error("conv_silu: bad argument"); return KTB200_EINVAL; }
    if (n_tokens <= 0) return KTB200_OK;
    const int C = channels, tile = n_tokens == n_seqs ? 1 : kConvTokens;
    const size_t esz = dtype == KTB200_TYPE_BF16 ? 2 : 4;
    const bool vec = C % 4 == 0 && in_stride % 4 == 0 && ssd_aligned(in, 4 * esz) && ssd_aligned(out, 4 * esz);
#define CONV_LAUNCH(VEC, TAPS)                                                                                                                                \
    conv_silu_kernel<T, VEC, TAPS><<<dim3((n_tokens + tile - 1) / tile, (C + kConvThreads * VEC - 1) / (kConvThreads * VEC)), kConvThreads, 0,                \
                                     (cudaStream_t)stream>>>((const T*)in, in_stride, (const T*)conv_w, (const T*)conv_b, taps, C, seq_of, seqs, seqs_stride, \
                                                             state, state_stride, conv_off, (T*)out, n_tokens, tile)
    SEQ_DISPATCH(dtype, {
        if (vec && taps == 4) CONV_LAUNCH(4, 4);
        else if (vec && taps == 3) CONV_LAUNCH(4, 3);
        else if (vec && taps == 2) CONV_LAUNCH(4, 2);
        else CONV_LAUNCH(1, 0);
    });
#undef CONV_LAUNCH
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}

extern "C" int ktb200_ssd_conv(const ktb200_ssd_params* c, void* xbc, int n_tokens, int dtype, void* stream) {
    if (ssd_bad(c) || !c->seq_of || !xbc) { set_error("ssd_conv: bad argument"); return KTB200_EINVAL; }
    const size_t esz = dtype == KTB200_TYPE_BF16 ? 2 : 4;
    return ktb200_conv_silu((const char*)c->proj + (size_t)c->xbc_off * esz, c->proj_stride, c->conv_w, c->conv_b, c->taps, c->heads * c->vdim + 2 * c->groups * c->state_size, c->seq_of,
                            c->seqs, c->seqs_stride, c->state, c->state_stride, (long)c->heads * c->state_size * c->vdim, xbc, n_tokens, c->n_seqs, dtype, stream);
}

/* whether ktb200_ssd_scan may run the chunked tensor-core form: bf16, a state size that is a multiple of 16 up to 256, 16-byte aligned rows */
extern "C" int ktb200_ssd_scan_uses_tensor_cores(int heads, int groups, int state_size, int vdim, int dtype) {
    return dtype == KTB200_TYPE_BF16 && heads > 0 && groups > 0 && heads % groups == 0 && state_size % 16 == 0 && state_size <= 256 && vdim % 8 == 0;
}

extern "C" int ktb200_ssd_scan(const ktb200_ssd_params* c, const void* xbc, float* y, int dtype, int allow_tensor_cores, void* stream) {
    if (ssd_bad(c) || !xbc || !y || c->state_size > kSsdWarps * kSsdRows) { set_error("ssd_scan: bad argument (state size <= %d)", kSsdWarps * kSsdRows); return KTB200_EINVAL; }
    if (c->n_seqs <= 0) return KTB200_OK;
    if (allow_tensor_cores && ktb200_ssd_scan_uses_tensor_cores(c->heads, c->groups, c->state_size, c->vdim, dtype) && ssd_aligned(xbc, 16)) {
        using B = __nv_bfloat16;
        const size_t smem = ssd_chunk_smem(c->state_size);
        const dim3 grid(c->n_seqs, c->heads, (c->vdim + kChunkCols - 1) / kChunkCols);
#define CHUNK_LAUNCH(MT)                                                                                                                                                       \
    do {                                                                                                                                                                       \
        GRANT_SMEM(ssd_chunk_kernel<MT>, smem);                                                                                                                                \
        ssd_chunk_kernel<MT><<<grid, 256, smem, (cudaStream_t)stream>>>((const B*)xbc, (const B*)c->proj + c->dt_off, c->proj_stride, c->dt_bias, c->a_log, c->d_skip, c->heads, \
                                                                        c->groups, c->state_size, c->vdim, c->seqs, c->seqs_stride, c->state, c->state_stride, y);            \
    } while (0)
        if (c->state_size <= 64) CHUNK_LAUNCH(1);
        else if (c->state_size <= 128) CHUNK_LAUNCH(2);
        else CHUNK_LAUNCH(4);
#undef CHUNK_LAUNCH
        KTB_LAUNCH_CHECK();
        return KTB200_OK;
    }
    const int N = c->state_size, rpt = (((N + kSsdWarps - 1) / kSsdWarps) + 3) & ~3, np = rpt * kSsdWarps;
    const size_t smem = ((size_t)2 * kSsdChunk * np + kSsdChunk * 34 + (size_t)kSsdChunk * kSsdWarps * 32) * sizeof(float);
    const dim3 grid(c->n_seqs, c->heads, (c->vdim + 31) / 32);
#define SSD_LAUNCH(ROWS)                                                                                                                                                 \
    SEQ_DISPATCH(dtype, {                                                                                                                                                \
        GRANT_SMEM((ssd_scan_kernel<T, ROWS>), smem);                                                                                                                    \
        ssd_scan_kernel<T, ROWS><<<grid, kSsdWarps * 32, smem, (cudaStream_t)stream>>>((const T*)xbc, (const T*)c->proj + c->dt_off, c->proj_stride, c->dt_bias, c->a_log, \
                                                                                      c->d_skip, c->heads, c->groups, N, c->vdim, c->seqs, c->seqs_stride, c->state,     \
                                                                                      c->state_stride, y);                                                              \
    })
    if (rpt <= 8) SSD_LAUNCH(8);
    else if (rpt <= 16) SSD_LAUNCH(16);
    else SSD_LAUNCH(32);
#undef SSD_LAUNCH
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}

extern "C" int ktb200_ssd_step(const ktb200_ssd_params* c, float* y, int dtype, void* stream) {
    if (ssd_bad(c) || !y) { set_error("ssd_step: bad argument"); return KTB200_EINVAL; }
    if (c->n_seqs <= 0) return KTB200_OK;
    const int N = c->state_size, dv = c->vdim;
    const long conv_off = (long)c->heads * N * dv;
    const bool vec = dv % 4 == 0 && c->state_stride % 4 == 0 && ssd_aligned(c->state, 16);
    // columns per CTA: a head's, or 32 when that leaves SMs idle; never more than 256 threads own
    int cpb = vec ? (dv + 3) / 4 * 4 : dv;
    if (cpb > 256) cpb = 256;
    if ((long)c->n_seqs * c->heads < 2 * 148 && cpb > 32) cpb = 32;
    const int tcol = vec ? cpb / 4 : cpb, rows_par = 256 / tcol;
    const size_t smem = ((size_t)cpb + 2 * N + (size_t)rows_par * cpb) * sizeof(float);
    if (smem > 200 * 1024) { set_error("ssd_step: state too large for shared memory"); return KTB200_EINVAL; }
    const dim3 grid(c->n_seqs, c->heads, (dv + cpb - 1) / cpb);
#define STEP_LAUNCH(VEC)                                                                                                                                                \
    SEQ_DISPATCH(dtype, {                                                                                                                                               \
        GRANT_SMEM((ssd_step_kernel<T, VEC>), smem);                                                                                                                    \
        ssd_step_kernel<T, VEC><<<grid, 256, smem, (cudaStream_t)stream>>>((const T*)c->proj, c->proj_stride, c->xbc_off, c->dt_off, (const T*)c->conv_w, (const T*)c->conv_b, \
                                                                          c->taps, c->dt_bias, c->a_log, c->d_skip, c->heads, c->groups, N, dv, c->seqs, c->seqs_stride,  \
                                                                          c->state, c->state_stride, conv_off, y, cpb);                                                \
    })
    if (vec) STEP_LAUNCH(4);
    else STEP_LAUNCH(1);
#undef STEP_LAUNCH
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}

extern "C" int ktb200_gated_group_norm(const float* y, const void* z, long z_stride, const void* weight, int groups, float eps, float out_scale, void* out, long out_stride, int n_tokens,
                                       int width, int dtype, void* stream) {
    if (!y || !z || !weight || !out || groups <= 0 || width <= 0 || width % groups || out_stride < width) { set_error("gated_group_norm: bad argument"); return KTB200_EINVAL; }
    if (n_tokens <= 0) return KTB200_OK;
    const int n = width / groups;
    const size_t smem = (size_t)n * sizeof(float), esz = dtype == KTB200_TYPE_BF16 ? 2 : 4;
    if (smem > 200 * 1024) { set_error("gated_group_norm: part too wide for shared memory"); return KTB200_EINVAL; }
    const int vec = n % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0 && ssd_aligned(y, 16) && ssd_aligned(z, 4 * esz) && ssd_aligned(out, 4 * esz) && ssd_aligned(weight, 4 * esz);
    const int threads = n >= 2048 ? 512 : (n >= 512 ? 256 : 128);
    SEQ_DISPATCH(dtype, {
        GRANT_SMEM(gated_group_norm_kernel<T>, smem);
        gated_group_norm_kernel<T><<<dim3(n_tokens, groups), threads, smem, (cudaStream_t)stream>>>(y, (const T*)z, z_stride, (const T*)weight, eps, out_scale, (T*)out, out_stride, n, vec);
    });
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}
