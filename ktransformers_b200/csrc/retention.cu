// Retention: linear attention whose matrix state per head decays by one fixed number per head, with rotated queries and keys, a unit-rms head
// output and an output gate (libktb200_seq.so).
//
//   S <- decay_h S + k v^T ;  o = S^T q ;  out = o / sqrt(mean_c(o_c^2) + eps) * silu(g)          per head; q, k turned, k times k_scale
//
//   ktb200_turn_table        the (cos, sin) pairs of a step's tokens, once for all layers of the same rotation
//   ktb200_retention_chunk   prompt portions in chunks on the tensor cores, all chunks in parallel (bf16)
//   ktb200_retention_scan    token by token on CUDA cores (fp32, sizes outside the tiles, short portions), o left for ktb200_gla_out
//   ktb200_retention_step    decode steps: rotation, recurrence, norm and gate in one launch, a head's column blocks as a thread-block cluster
//
// State row of a sequence and layer (fp32): S [heads][dim][vdim], read from the row seqs[2][s] (or zeros when -1) and written to the row seqs[3][s].
// Storage type T (bf16 or float) for projections and outputs; turned queries and keys, decays, the state and everything read from it are fp32 (on
// the tensor cores: two bf16 terms per operand).
#include <cooperative_groups.h>
#include <cuda_bf16.h>

#include "common.cuh"
#include "seq_common.cuh"
#include "mma_tile.cuh"

namespace ktb {

struct Retention {
    const void* proj;
    long stride;
    int q_off, k_off, v_off, g_off, H, d, dv, rot_dims, layout;
    const float2* turn;      // [T][rot_dims / 2]
    float k_scale;
    const float *decay, *decay_low, *log2_decay;
    float eps;
    const int* seqs;
    int seqs_stride, n_seqs;
    float* state;
    long state_stride;
};

// S decay + u with the decay as the sum of two floats in 32-bit runs: what its rounding leaves out would add up along the tokens
template <typename T> __device__ __forceinline__ float kept(float S, float decay, float low, float u) { return fmaf(decay, S, sizeof(T) == 4 ? fmaf(low, S, u) : u); }

__global__ void turn_table_kernel(const int* __restrict__ pos, const double* __restrict__ inv_freq, int pairs, float2* __restrict__ turn, long n) {
    for (long i = blockIdx.x * (long)blockDim.x + threadIdx.x; i < n; i += (long)gridDim.x * blockDim.x) {
        const long t = i / pairs;
        double sn, cs;
        sincos((double)pos[t] * inv_freq[i - t * pairs], &sn, &cs);
        turn[i] = make_float2((float)cs, (float)sn);
    }
}

// column c of a head's row after the rotation; tr: the token's pairs
template <typename T>
__device__ __forceinline__ float turned(const T* __restrict__ row, int c, int rot_dims, int layout, const float2* __restrict__ tr) {
    const float v = to_f(row[c]);
    if (c >= rot_dims) return v;
    const float other = to_f(row[rot_partner(c, rot_dims, layout)]);
    const int half = rot_dims >> 1;
    const bool second = layout == kRotHalves ? c >= half : (c & 1);
    const float2 cs = tr[layout == kRotHalves ? (second ? c - half : c) : (c >> 1)];
    return second ? v * cs.x + other * cs.y : v * cs.x - other * cs.y;
}

// ------------------------------------------------------------------------------------------------ token by token
// grid (portions, heads, column blocks of 32 value columns); 8 warps; thread (warp w, lane) keeps S[i][col] for a contiguous run of key rows i in
// registers.  Tokens run in order in chunks of kRetChunk staged in shared memory, the next chunk's inputs fetched (and turned) while the current one
// runs; per token every warp leaves its part of o in shared memory, summed in warp order once per chunk.
constexpr int kRetChunk = 16, kRetWarps = 8, kRetRows = 32;      // dim <= 256
template <typename T, int ROWS>
__global__ void __launch_bounds__(256, 2) retention_scan_kernel(const Retention a, float* __restrict__ o_out) {
    extern __shared__ __align__(16) float sm[];
    const int d = a.d, dv = a.dv, H = a.H, half = a.rot_dims >> 1;
    const int rpt = (((d + kRetWarps - 1) / kRetWarps) + 3) & ~3, dp = rpt * kRetWarps;
    float* qs = sm;                             // [chunk][dp]
    float* ks = qs + kRetChunk * dp;            // [chunk][dp]
    float* vs = ks + kRetChunk * dp;            // [chunk][32]
    float* part = vs + kRetChunk * 32;          // [chunk][warps][32]
    const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * 32;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, col = c0 + lane;
    const int start = a.seqs[s], len = a.seqs[a.seqs_stride + s], rd = a.seqs[2 * a.seqs_stride + s], wr = a.seqs[3 * a.seqs_stride + s];
    const T* proj = (const T*)a.proj;
    const float keep = a.decay[h], low = a.decay_low[h];
    float S[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; r++) {
        const int i = warp * rpt + r;
        S[r] = (rd >= 0 && r < rpt && i < d && col < dv) ? a.state[(long)rd * a.state_stride + ((long)h * d + i) * dv + col] : 0.f;
    }
    constexpr int E = kRetChunk * ROWS * kRetWarps / 256;      // staged values per thread and array, at most
    float rq[E], rk[E], rv[2];
    auto fetch = [&](int t0) {
        const int nt = min(kRetChunk, len - t0);
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = threadIdx.x + e * 256;
            rq[e] = rk[e] = 0.f;
            if (i < nt * dp) {
                const int tt = i / dp, c = i - tt * dp;
                const long t = (long)(start + t0 + tt);
                if (c < d) {
                    rq[e] = turned(proj + t * a.stride + a.q_off + (long)h * d, c, a.rot_dims, a.layout, a.turn + t * half);
                    rk[e] = turned(proj + t * a.stride + a.k_off + (long)h * d, c, a.rot_dims, a.layout, a.turn + t * half) * a.k_scale;
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int i = threadIdx.x + e * 256, c = c0 + (i & 31);
            rv[e] = (i < nt * 32 && c < dv) ? to_f(proj[(long)(start + t0 + (i >> 5)) * a.stride + a.v_off + (long)h * dv + c]) : 0.f;
        }
    };
    if (len > 0) fetch(0);
    for (int t0 = 0; t0 < len; t0 += kRetChunk) {
        const int nt = min(kRetChunk, len - t0);
        __syncthreads();      // the previous chunk is consumed
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = threadIdx.x + e * 256;
            if (i < nt * dp) { qs[i] = rq[e]; ks[i] = rk[e]; }
        }
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int i = threadIdx.x + e * 256;
            if (i < nt * 32) vs[i] = rv[e];
        }
        __syncthreads();
        if (t0 + kRetChunk < len) fetch(t0 + kRetChunk);
#pragma unroll 2
        for (int tt = 0; tt < nt; tt++) {
            const float v = vs[tt * 32 + lane];
            const float4* qr = reinterpret_cast<const float4*>(qs + tt * dp + warp * rpt);
            const float4* kr = reinterpret_cast<const float4*>(ks + tt * dp + warp * rpt);
            float o0 = 0.f, o1 = 0.f;
#pragma unroll
            for (int r4 = 0; r4 < ROWS / 4; r4++) {
                if (4 * r4 < rpt) {
                    const float4 k = kr[r4], q = qr[r4];
                    S[4 * r4] = kept<T>(S[4 * r4], keep, low, k.x * v);
                    o0 = fmaf(S[4 * r4], q.x, o0);
                    S[4 * r4 + 1] = kept<T>(S[4 * r4 + 1], keep, low, k.y * v);
                    o1 = fmaf(S[4 * r4 + 1], q.y, o1);
                    S[4 * r4 + 2] = kept<T>(S[4 * r4 + 2], keep, low, k.z * v);
                    o0 = fmaf(S[4 * r4 + 2], q.z, o0);
                    S[4 * r4 + 3] = kept<T>(S[4 * r4 + 3], keep, low, k.w * v);
                    o1 = fmaf(S[4 * r4 + 3], q.w, o1);
                }
            }
            part[(tt * kRetWarps + warp) * 32 + lane] = o0 + o1;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nt * 32; i += blockDim.x) {
            const int tt = i >> 5, c = c0 + (i & 31);
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < kRetWarps; w++) o += part[(tt * kRetWarps + w) * 32 + (i & 31)];
            if (c < dv) o_out[((long)(start + t0 + tt) * H + h) * dv + c] = o;
        }
    }
    if (wr >= 0) {
#pragma unroll
        for (int r = 0; r < ROWS; r++) {
            const int i = warp * rpt + r;
            if (r < rpt && i < d && col < dv) a.state[(long)wr * a.state_stride + ((long)h * d + i) * dv + col] = S[r];
        }
    }
}

// ------------------------------------------------------------------------------------------------ chunks on the tensor cores (bf16)
// With fixed decays the states along a portion follow from one pass over the sums of its parts, so all parts of all portions and heads run at once:
//   1. chunk_state   turns q and k, and per span of 128 tokens:  U_s = sum_j decay^(n - 1 - j) k_j v_j^T                        (n tokens in the span)
//   2. carry         S_s = the state ahead of span s: S_(s+1) = decay^n S_s + U_s, elementwise along the portion's spans; S_s replaces U_s
//   3. chunk_out     chunks of 64 tokens, c tokens behind their span's start (0 or 64):
//                    o_i = decay^(c + i + 1) S_s^T q_i + sum over the span's keys j up to i of decay^(i - j) (q_i . k_j) v_j, then norm and gate
// m16n8k16 bf16 MMAs with fp32 accumulators; v is bf16 as it comes, every other operand (turned q and k, weighted k and scores, S) enters as the
// sum of two bf16 terms hi + lo (about 16 bits of mantissa), products of two such operands as hi hi + hi lo + lo hi.
// Workspace: per (span, head) dim * vdim fp32 of U, then in the same bytes S as groups of 8 columns [8 hi | 8 lo]; per (token, head) the turned q
// and the turned and scaled k as rows [dim hi | dim lo].
constexpr int kRetQ = 64, kRetSpan = 2 * kRetQ;
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
// which portion tile b of `per` tokens belongs to: {portion or -1, first token's offset in the portion, tokens, the portion's first span}
__device__ __forceinline__ void find_chunk(const int* __restrict__ seqs, int stride, int n_seqs, int b, int per, int (&info)[4]) {
    info[0] = -1;
    int spans = 0;
    for (int s = 0; s < n_seqs; s++) {
        const int len = seqs[stride + s], nt = (len + per - 1) / per;
        if (b < nt) {
            info[0] = s;
            info[1] = b * per;
            info[2] = min(per, len - b * per);
            info[3] = spans;
            return;
        }
        b -= nt;
        spans += (len + kRetSpan - 1) / kRetSpan;
    }
}
// The nt rows of a head (first row `src`, rows `stride` apart; up to 64 rows as zeros behind them), turned: sink(row, column, four neighbouring columns).
// Where the pair halves are runs of four columns: four pairs at a time, the loads of AHEAD such units in flight together.
template <int AHEAD, class Sink>
__device__ __forceinline__ void turned_rows(const __nv_bfloat16* __restrict__ src, long stride, int nt, int d, int rot_dims, int layout, const float2* __restrict__ turn, Sink sink) {
    const int half = rot_dims >> 1;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    if (layout == kRotHalves && half % 4 == 0 && rot_dims > 0) {
        const int pairs = half / 4, per = pairs + (d - rot_dims) / 4;      // units of a row: four pairs, or four columns that pass (d - rot_dims is a multiple of 4 here)
        for (int i0 = threadIdx.x; i0 < kRetQ * per; i0 += AHEAD * blockDim.x) {
            uint2 p[AHEAD], q[AHEAD];
            float4 c0[AHEAD], c1[AHEAD];
#pragma unroll
            for (int k = 0; k < AHEAD; k++) {
                const int i = i0 + k * blockDim.x, r = i / per, u = i - r * per;
                p[k] = q[k] = make_uint2(0, 0);
                c0[k] = c1[k] = zero;
                if (r < nt && i < kRetQ * per) {
                    const __nv_bfloat16* row = src + (long)r * stride;
                    if (u < pairs) {
                        p[k] = *reinterpret_cast<const uint2*>(row + u * 4);
                        q[k] = *reinterpret_cast<const uint2*>(row + half + u * 4);
                        c0[k] = *reinterpret_cast<const float4*>(turn + (long)r * half + u * 4);
                        c1[k] = *reinterpret_cast<const float4*>(turn + (long)r * half + u * 4 + 2);
                    } else {
                        p[k] = *reinterpret_cast<const uint2*>(row + rot_dims + (u - pairs) * 4);
                    }
                }
            }
#pragma unroll
            for (int k = 0; k < AHEAD; k++) {
                const int i = i0 + k * blockDim.x, r = i / per, u = i - r * per;
                if (i >= kRetQ * per) break;
                const float4 a = make_float4(__uint_as_float(p[k].x << 16), __uint_as_float(p[k].x & 0xffff0000u), __uint_as_float(p[k].y << 16), __uint_as_float(p[k].y & 0xffff0000u));
                if (u < pairs) {
                    const float4 b = make_float4(__uint_as_float(q[k].x << 16), __uint_as_float(q[k].x & 0xffff0000u), __uint_as_float(q[k].y << 16), __uint_as_float(q[k].y & 0xffff0000u));
                    sink(r, u * 4, make_float4(a.x * c0[k].x - b.x * c0[k].y, a.y * c0[k].z - b.y * c0[k].w, a.z * c1[k].x - b.z * c1[k].y, a.w * c1[k].z - b.w * c1[k].w));
                    sink(r, half + u * 4, make_float4(b.x * c0[k].x + a.x * c0[k].y, b.y * c0[k].z + a.y * c0[k].w, b.z * c1[k].x + a.z * c1[k].y, b.w * c1[k].z + a.w * c1[k].w));
                } else {
                    sink(r, rot_dims + (u - pairs) * 4, a);
                }
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < kRetQ * (d / 4); i += blockDim.x) {
        const int r = i / (d / 4), c = (i - r * (d / 4)) * 4;
        const __nv_bfloat16* row = src + (long)r * stride;
        const float2* tr = turn + (long)r * half;
        sink(r, c, r < nt ? make_float4(turned(row, c, rot_dims, layout, tr), turned(row, c + 1, rot_dims, layout, tr), turned(row, c + 2, rot_dims, layout, tr), turned(row, c + 3, rot_dims, layout, tr)) : zero);
    }
}
// four columns times w as two bf16 terms, the low ones `low` elements behind the high ones
__device__ __forceinline__ void put_split(__nv_bfloat16* hi, int low, float4 v, float w) {
    uint32_t h0, l0, h1, l1;
    split2(v.x * w, v.y * w, h0, l0);
    split2(v.z * w, v.w * w, h1, l1);
    *reinterpret_cast<uint2*>(hi) = make_uint2(h0, h1);
    *reinterpret_cast<uint2*>(hi + low) = make_uint2(l0, l1);
}
__device__ __forceinline__ void fetch_rows(__nv_bfloat16* dst, int ld, const __nv_bfloat16* __restrict__ src, long stride, int nt, int n) {      // nt of 64 rows of n columns, the rest zeros
    const int pieces = n >> 3;
    for (int i = threadIdx.x; i < kRetQ * pieces; i += blockDim.x) {
        const int r = i / pieces, c = (i - r * pieces) * 8;
        cp_async16(dst + r * ld + c, src + (long)(r < nt ? r : 0) * stride + c, r < nt);
    }
}

// grid (spans, heads), 8 warps; a unit of work is 16 key rows x up to 64 value columns of U, at most two per warp
__global__ void __launch_bounds__(256, 2) retention_chunk_state_kernel(const Retention a, float* __restrict__ ws, __nv_bfloat16* __restrict__ q_rows, __nv_bfloat16* __restrict__ k_rows) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ int info[4];
    __shared__ float row_w[kRetSpan];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, tq = lane & 3, h = blockIdx.y;
    const int d = a.d, dv = a.dv, ldk = d + 8, ldv = dv + 8;
    if (tid == 0) find_chunk(a.seqs, a.seqs_stride, a.n_seqs, blockIdx.x, kRetSpan, info);
    __syncthreads();
    if (info[0] < 0) return;
    const int n = info[2];
    const long t0 = a.seqs[info[0]] + info[1];
    __nv_bfloat16* Kh = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* Kl = Kh + kRetQ * ldk;
    __nv_bfloat16* Vs = Kl + kRetQ * ldk;
    const __nv_bfloat16* proj = (const __nv_bfloat16*)a.proj;
    if (tid < kRetSpan) row_w[tid] = tid < n ? exp2f((float)(n - 1 - tid) * a.log2_decay[h]) : 0.f;
    const int d16 = d >> 4, dv16 = dv >> 4, cgroups = (dv16 + 3) >> 2;
    float acc[2][8][4];
#pragma unroll
    for (int k = 0; k < 2; k++)
#pragma unroll
        for (int m = 0; m < 8; m++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[k][m][e] = 0.f;
    for (int part = 0; part * kRetQ < n; part++) {
        const long t1 = t0 + part * kRetQ;
        const int nt = min(kRetQ, n - part * kRetQ), k16 = (nt + 15) >> 4;
        __syncthreads();      // row_w is there; the first half is consumed
        fetch_rows(Vs, ldv, proj + t1 * a.stride + a.v_off + (long)h * dv, a.stride, nt, dv);
        const float2* turn = a.turn + t1 * (a.rot_dims >> 1);
        const __nv_bfloat16* rows = proj + t1 * a.stride + (long)h * d;
        turned_rows<2>(rows + a.k_off, a.stride, nt, d, a.rot_dims, a.layout, turn, [&](int r, int c, float4 v) {
            if (r < nt) put_split(k_rows + ((t1 + r) * a.H + h) * (2L * d) + c, d, v, a.k_scale);
            put_split(Kh + r * ldk + c, kRetQ * ldk, v, r < nt ? a.k_scale * row_w[part * kRetQ + r] : 0.f);
        });
        turned_rows<2>(rows + a.q_off, a.stride, nt, d, a.rot_dims, a.layout, turn, [&](int r, int c, float4 v) {
            if (r < nt) put_split(q_rows + ((t1 + r) * a.H + h) * (2L * d) + c, d, v, 1.0f);
        });
        cp_async_wait_all();
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const int unit = warp + 8 * k;
            if (unit < d16 * cgroups) {
                const int r0 = (unit / cgroups) * 16, v0 = (unit % cgroups) * 4;
                for (int kk = 0; kk < k16; kk++) {
                    uint32_t ah[4], al[4];
                    const int at = (kk * 16 + (lane & 7) + 8 * (lane >> 4)) * ldk + r0 + 8 * ((lane >> 3) & 1);
                    ldmatrix_x4_trans(ah, Kh + at);
                    ldmatrix_x4_trans(al, Kl + at);
#pragma unroll
                    for (int vp = 0; vp < 4; vp++) {
                        if (v0 + vp < dv16) {
                            uint32_t b[4];
                            ldmatrix_x4_trans(b, Vs + (kk * 16 + (lane & 15)) * ldv + (v0 + vp) * 16 + 8 * (lane >> 4));
                            mma_bf16_16816(acc[k][2 * vp], ah, b[0], b[1]);
                            mma_bf16_16816(acc[k][2 * vp + 1], ah, b[2], b[3]);
                            mma_bf16_16816(acc[k][2 * vp], al, b[0], b[1]);
                            mma_bf16_16816(acc[k][2 * vp + 1], al, b[2], b[3]);
                        }
                    }
                }
            }
        }
    }
    float* U = ws + ((long)blockIdx.x * a.H + h) * d * dv;
#pragma unroll
    for (int k = 0; k < 2; k++) {
        const int unit = warp + 8 * k;
        if (unit < d16 * cgroups) {
            const int r0 = (unit / cgroups) * 16, v0 = (unit % cgroups) * 4;
#pragma unroll
            for (int m = 0; m < 8; m++) {
                const int c = v0 * 16 + m * 8 + 2 * tq;
                if (c < dv) {
                    *reinterpret_cast<float2*>(U + (long)(r0 + gq) * dv + c) = make_float2(acc[k][m][0], acc[k][m][1]);
                    *reinterpret_cast<float2*>(U + (long)(r0 + gq + 8) * dv + c) = make_float2(acc[k][m][2], acc[k][m][3]);
                }
            }
        }
    }
}

// grid (blocks of 128 x 8 elements, heads, portions); a thread carries eight neighbouring columns along the portion's spans, kCarryAhead of whose sums
// are in flight
constexpr int kCarryAhead = 4;
__global__ void __launch_bounds__(128) retention_carry_kernel(const Retention a, float* __restrict__ ws) {
    const int s = blockIdx.z, h = blockIdx.y;
    const long n = (long)a.d * a.dv, i = (blockIdx.x * 128L + threadIdx.x) * 8;
    if (i >= n) return;
    long first = 0;
    for (int k = 0; k < s; k++) first += (a.seqs[a.seqs_stride + k] + kRetSpan - 1) / kRetSpan;
    const int len = a.seqs[a.seqs_stride + s], rd = a.seqs[2 * a.seqs_stride + s], wr = a.seqs[3 * a.seqs_stride + s], spans = (len + kRetSpan - 1) / kRetSpan;
    const float l2 = a.log2_decay[h], full = exp2f((float)kRetSpan * l2);
    float4 S0 = make_float4(0.f, 0.f, 0.f, 0.f), S1 = S0;
    if (rd >= 0) {
        const float* p = a.state + (long)rd * a.state_stride + (long)h * n + i;
        S0 = load4(p);
        S1 = load4(p + 4);
    }
    const long step = (long)a.H * n;
    float* U = ws + (first * a.H + h) * n + i;
    for (int c0 = 0; c0 < spans; c0 += kCarryAhead) {
        float4 u[kCarryAhead][2];
#pragma unroll
        for (int k = 0; k < kCarryAhead; k++)
            if (c0 + k < spans) {
                u[k][0] = load4(U + (c0 + k) * step);
                u[k][1] = load4(U + (c0 + k) * step + 4);
            }
#pragma unroll
        for (int k = 0; k < kCarryAhead; k++) {
            const int c = c0 + k;
            if (c >= spans) break;
            uint4 hi, lo;
            split2(S0.x, S0.y, hi.x, lo.x);
            split2(S0.z, S0.w, hi.y, lo.y);
            split2(S1.x, S1.y, hi.z, lo.z);
            split2(S1.z, S1.w, hi.w, lo.w);
            uint4* o = reinterpret_cast<uint4*>(U + c * step);
            o[0] = hi;
            o[1] = lo;
            const float f = c + 1 < spans ? full : exp2f((float)(len - c * kRetSpan) * l2);
            S0 = make_float4(fmaf(f, S0.x, u[k][0].x), fmaf(f, S0.y, u[k][0].y), fmaf(f, S0.z, u[k][0].z), fmaf(f, S0.w, u[k][0].w));
            S1 = make_float4(fmaf(f, S1.x, u[k][1].x), fmaf(f, S1.y, u[k][1].y), fmaf(f, S1.z, u[k][1].z), fmaf(f, S1.w, u[k][1].w));
        }
    }
    if (wr >= 0) {
        float* p = a.state + (long)wr * a.state_stride + (long)h * n + i;
        store4(p, S0);
        store4(p + 4, S1);
    }
}

// grid (chunks, heads), 8 warps: warp w has the chunk's tokens 16 (w & 3) .. + 15 and one half of the value columns.  Shared memory: Q hi, lo | K hi,
// lo | V | weighted scores hi, lo; ahead of the keys the state's first 64 key rows where K goes and the others where V and the scores go.  The score
// tiles of 16 tokens are shared out between their two warps and pass through shared memory.
constexpr int kRetLdA = kRetQ + 8;
__host__ __device__ static inline int ret_k_elems(int d, int dv) { return 2 * kRetQ * ((d > dv ? d : dv) + 8); }      // (K rows are d columns, state rows dv)
static size_t ret_out_smem(int d, int dv) {
    const size_t va = (size_t)kRetQ * (dv + 8) + 2 * kRetQ * kRetLdA, state = (size_t)2 * kRetQ * (dv + 8);
    return ((size_t)2 * kRetQ * (d + 8) + ret_k_elems(d, dv) + (d > kRetQ && state > va ? state : va)) * sizeof(__nv_bfloat16);
}
template <int D16MAX, int DV16MAX>
__global__ void __launch_bounds__(256, 2) retention_chunk_out_kernel(const Retention a, const float* __restrict__ ws, const __nv_bfloat16* __restrict__ q_rows,
                                                                      const __nv_bfloat16* __restrict__ k_rows, __nv_bfloat16* __restrict__ out) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    constexpr int VT = (DV16MAX + 1) / 2;      // 16-column tiles per warp
    __shared__ int info[4];
    __shared__ float pw[kRetSpan + 1], row_sq[2][kRetQ];      // powers of the decay; squares of the two column halves
    const int tid = threadIdx.x, lane = tid & 31, rg = (tid >> 5) & 3, side = tid >> 7, gq = lane >> 2, tq = lane & 3, h = blockIdx.y;
    const int d = a.d, dv = a.dv, d16 = d >> 4, dv16 = dv >> 4, ldk = d + 8, ldv = dv + 8;
    if (tid == 0) find_chunk(a.seqs, a.seqs_stride, a.n_seqs, blockIdx.x, kRetQ, info);
    if (tid <= kRetSpan) pw[tid] = exp2f((float)tid * a.log2_decay[h]);
    __syncthreads();
    if (info[0] < 0) return;
    const int nt = info[2], behind = info[1] % kRetSpan;      // tokens of the span ahead of this chunk
    const long t0 = a.seqs[info[0]] + info[1];
    const bool has_state = info[1] >= kRetSpan || a.seqs[2 * a.seqs_stride + info[0]] >= 0;
    __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* Ql = Qh + kRetQ * ldk;
    __nv_bfloat16* Kh = Ql + kRetQ * ldk;
    __nv_bfloat16* Kl = Kh + kRetQ * ldk;
    __nv_bfloat16* Vs = Kh + ret_k_elems(d, dv);
    __nv_bfloat16* Ah = Vs + kRetQ * ldv;
    __nv_bfloat16* Al = Ah + kRetQ * kRetLdA;
    const __nv_bfloat16* proj = (const __nv_bfloat16*)a.proj;
    const int groups = dv >> 3, kp = d >> 3;
    if (has_state) {      // key rows in pieces of 64, groups of 8 columns [8 hi | 8 lo]
        const __nv_bfloat16* Sg = reinterpret_cast<const __nv_bfloat16*>(ws + (((long)info[3] + info[1] / kRetSpan) * a.H + h) * d * dv);
        for (int i = tid; i < d * groups; i += 256) {
            const int r = i / groups, g = i - r * groups;
            const __nv_bfloat16* src = Sg + (long)i * 16;
            __nv_bfloat16* dst = (r < kRetQ ? Kh : Vs) + (r & (kRetQ - 1)) * ldv + g * 8;
            cp_async16(dst, src, true);
            cp_async16(dst + kRetQ * ldv, src + 8, true);
        }
    }
    auto fetch_planes = [&](__nv_bfloat16* hi, const __nv_bfloat16* rows, int n) {      // n of 64 rows [d hi | d lo], the rest zeros
        for (int i = tid; i < kRetQ * kp; i += 256) {
            const int r = i / kp, c = (i - r * kp) * 8;
            const __nv_bfloat16* src = rows + (long)(r < n ? r : 0) * a.H * (2 * d) + c;
            cp_async16(hi + r * ldk + c, src, r < n);
            cp_async16(hi + (kRetQ + r) * ldk + c, src + d, r < n);
        }
    };
    fetch_planes(Qh, q_rows + (t0 * a.H + h) * (2L * d), nt);
    const bool live = rg * 16 < nt;
    const int v0 = side * ((dv16 + 1) >> 1), v1 = side ? dv16 : (dv16 + 1) >> 1;      // this warp's column tiles
    float Y[2 * VT][4];
#pragma unroll
    for (int n = 0; n < 2 * VT; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) Y[n][e] = 0.f;
    const int qat = (rg * 16 + (lane & 15)) * ldk + 8 * (lane >> 4);
    const int iA = rg * 16 + gq, iB = iA + 8;
    if (has_state) {
        cp_async_wait_all();
        __syncthreads();
        if (live) {
#pragma unroll 2
            for (int kk = 0; kk < d16; kk++) {
                uint32_t qh[4], ql[4];
                ldmatrix_x4(qh, Qh + qat + kk * 16);
                ldmatrix_x4(ql, Ql + qat + kk * 16);
                const __nv_bfloat16* Sk = (kk < 4 ? Kh : Vs) + ((kk & 3) * 16 + (lane & 15)) * ldv + 8 * (lane >> 4);
#pragma unroll
                for (int vp = 0; vp < VT; vp++) {
                    if (v0 + vp < v1) {
                        uint32_t bh[4], bl[4];
                        ldmatrix_x4_trans(bh, Sk + (v0 + vp) * 16);
                        ldmatrix_x4_trans(bl, Sk + kRetQ * ldv + (v0 + vp) * 16);
                        mma_bf16_16816(Y[2 * vp], qh, bh[0], bh[1]);
                        mma_bf16_16816(Y[2 * vp + 1], qh, bh[2], bh[3]);
                        mma_bf16_16816(Y[2 * vp], ql, bh[0], bh[1]);
                        mma_bf16_16816(Y[2 * vp + 1], ql, bh[2], bh[3]);
                        mma_bf16_16816(Y[2 * vp], qh, bl[0], bl[1]);
                        mma_bf16_16816(Y[2 * vp + 1], qh, bl[2], bl[3]);
                    }
                }
            }
        }
        const float fA = pw[min(kRetSpan, behind + iA + 1)], fB = pw[min(kRetSpan, behind + iB + 1)];
#pragma unroll
        for (int n = 0; n < 2 * VT; n++) {
            Y[n][0] *= fA;
            Y[n][1] *= fA;
            Y[n][2] *= fB;
            Y[n][3] *= fB;
        }
    }
    // the span's keys: the 64 tokens ahead of this chunk when it is the second of its span, then the chunk's own
    for (int back = behind; back >= 0; back -= kRetQ) {
        const long t1 = t0 - back;
        const int kt = back ? kRetQ : nt;
        if (has_state || back != behind) __syncthreads();      // the state, or the keys and scores ahead, are consumed
        fetch_rows(Vs, ldv, proj + t1 * a.stride + a.v_off + (long)h * dv, a.stride, kt, dv);
        fetch_planes(Kh, k_rows + (t1 * a.H + h) * (2L * d), kt);
        cp_async_wait_all();
        __syncthreads();
        const int tiles = back ? kRetQ / 16 : rg + 1;      // key tiles of 16 that the warp's tokens see
        if (live) {
            for (int np = side; np < tiles; np += 2) {
                float G[2][4];
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) G[n][e] = 0.f;
                const int kat = (np * 16 + (lane & 7) + 8 * (lane >> 4)) * ldk + 8 * ((lane >> 3) & 1);
#pragma unroll
                for (int kk = 0; kk < D16MAX; kk++) {
                    if (kk < d16) {
                        uint32_t qh[4], ql[4], kh[4], kl[4];
                        ldmatrix_x4(qh, Qh + qat + kk * 16);
                        ldmatrix_x4(ql, Ql + qat + kk * 16);
                        ldmatrix_x4(kh, Kh + kat + kk * 16);
                        ldmatrix_x4(kl, Kl + kat + kk * 16);
                        mma_bf16_16816(G[0], qh, kh[0], kh[1]);
                        mma_bf16_16816(G[1], qh, kh[2], kh[3]);
                        mma_bf16_16816(G[0], ql, kh[0], kh[1]);
                        mma_bf16_16816(G[1], ql, kh[2], kh[3]);
                        mma_bf16_16816(G[0], qh, kl[0], kl[1]);
                        mma_bf16_16816(G[1], qh, kl[2], kl[3]);
                    }
                }
#pragma unroll
                for (int n = 0; n < 2; n++) {
                    const int j = np * 16 + n * 8 + 2 * tq;
#pragma unroll
                    for (int e = 0; e < 4; e += 2) {
                        const int i = back + (e ? iB : iA);
                        uint32_t hi, lo;
                        split2(i >= j ? G[n][e] * pw[i - j] : 0.f, i > j ? G[n][e + 1] * pw[max(0, i - j - 1)] : 0.f, hi, lo);
                        *reinterpret_cast<uint32_t*>(Ah + (e ? iB : iA) * kRetLdA + j) = hi;
                        *reinterpret_cast<uint32_t*>(Al + (e ? iB : iA) * kRetLdA + j) = lo;
                    }
                }
            }
        }
        __syncthreads();
        if (live) {
            for (int np = 0; np < tiles; np++) {
                uint32_t gh[4], gl[4];
                const int at = (rg * 16 + (lane & 15)) * kRetLdA + np * 16 + 8 * (lane >> 4);
                ldmatrix_x4(gh, Ah + at);
                ldmatrix_x4(gl, Al + at);
#pragma unroll
                for (int vp = 0; vp < VT; vp++) {
                    if (v0 + vp < v1) {
                        uint32_t b[4];
                        ldmatrix_x4_trans(b, Vs + (np * 16 + (lane & 15)) * ldv + (v0 + vp) * 16 + 8 * (lane >> 4));
                        mma_bf16_16816(Y[2 * vp], gh, b[0], b[1]);
                        mma_bf16_16816(Y[2 * vp + 1], gh, b[2], b[3]);
                        mma_bf16_16816(Y[2 * vp], gl, b[0], b[1]);
                        mma_bf16_16816(Y[2 * vp + 1], gl, b[2], b[3]);
                    }
                }
            }
        }
    }
    float sA = 0.f, sB = 0.f;      // (tiles beyond the warp's own hold zeros)
#pragma unroll
    for (int n = 0; n < 2 * VT; n++) {
        sA += Y[n][0] * Y[n][0] + Y[n][1] * Y[n][1];
        sB += Y[n][2] * Y[n][2] + Y[n][3] * Y[n][3];
    }
    sA += __shfl_xor_sync(0xffffffffu, sA, 1);
    sA += __shfl_xor_sync(0xffffffffu, sA, 2);
    sB += __shfl_xor_sync(0xffffffffu, sB, 1);
    sB += __shfl_xor_sync(0xffffffffu, sB, 2);
    if (tq == 0) {
        row_sq[side][iA] = sA;
        row_sq[side][iB] = sB;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int i = r ? iB : iA;
        if (i >= nt) continue;
        const float inv = 1.0f / sqrtf((row_sq[0][i] + row_sq[1][i]) / (float)dv + a.eps);
        const __nv_bfloat16* g = proj + (t0 + i) * a.stride + a.g_off + (long)h * dv;
        __nv_bfloat16* o = out + ((t0 + i) * a.H + h) * (long)dv;
#pragma unroll
        for (int n = 0; n < 2 * VT; n++) {
            const int c = v0 * 16 + n * 8 + 2 * tq;
            if (c < v1 * 16) {
                const uint32_t u = *reinterpret_cast<const uint32_t*>(g + c);
                *reinterpret_cast<uint32_t*>(o + c) =
                    pack_bf16(Y[n][2 * r] * inv * silu_for<__nv_bfloat16>(__uint_as_float(u << 16)), Y[n][2 * r + 1] * inv * silu_for<__nv_bfloat16>(__uint_as_float(u & 0xffff0000u)));
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ one token per portion
// grid (portions, heads, column blocks of `cpb` columns); the column blocks of a head are a thread-block cluster, which adds up the squares of the
// head's output over distributed shared memory.  A thread owns VEC columns of every `rows_par`-th state row, kRetStepRows of which it requests
// before q and k are turned.
constexpr int kRetStepRows = 8, kRetMaxBlocks = 8;
template <typename T, int VEC>
__global__ void __launch_bounds__(256) retention_step_kernel(const Retention a, T* __restrict__ out, int cpb) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32], squares;
    const int d = a.d, dv = a.dv, half = a.rot_dims >> 1;
    float* qs = sm;                        // [d]
    float* ks = qs + ((d + 3) & ~3);       // [d]
    float* os = ks + ((d + 3) & ~3);       // [cpb]
    float* part = os + ((cpb + 3) & ~3);   // [rows_par][cpb]
    const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * cpb, ncol = min(cpb, dv - c0);
    const int tcol = cpb / VEC, rows_par = blockDim.x / tcol, tc = threadIdx.x % tcol, tr = threadIdx.x / tcol, cc = tc * VEC;
    const bool mine = tr < rows_par && cc < ncol;
    const long t = a.seqs[s];
    const int rd = a.seqs[2 * a.seqs_stride + s], wr = a.seqs[3 * a.seqs_stride + s];
    const float* Sr = a.state + (long)rd * a.state_stride + (long)h * d * dv + c0 + cc;
    float* Sw = a.state + (long)wr * a.state_stride + (long)h * d * dv + c0 + cc;
    float v[kRetStepRows][VEC];
    auto request = [&](int base) {
#pragma unroll
        for (int k = 0; k < kRetStepRows; k++) {
            const int n = base + k * rows_par + tr;
            if (mine && rd >= 0 && n < d) {
                if (VEC == 4) {
                    const float4 u = load4(Sr + (long)n * dv);
                    v[k][0] = u.x; v[k][VEC > 1 ? 1 : 0] = u.y; v[k][VEC > 2 ? 2 : 0] = u.z; v[k][VEC > 3 ? 3 : 0] = u.w;
                } else {
                    v[k][0] = Sr[(long)n * dv];
                }
            } else {
#pragma unroll
                for (int e = 0; e < VEC; e++) v[k][e] = 0.f;
            }
        }
    };
    request(0);
    const T* row = (const T*)a.proj + t * a.stride;
    float x[VEC], y[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) {
        x[e] = mine && cc + e < ncol ? to_f(row[a.v_off + (long)h * dv + c0 + cc + e]) : 0.f;
        y[e] = 0.f;
    }
    for (int i = threadIdx.x; i < 2 * d; i += blockDim.x) {
        const bool is_k = i >= d;
        const int c = is_k ? i - d : i;
        const float u = turned(row + (is_k ? a.k_off : a.q_off) + (long)h * d, c, a.rot_dims, a.layout, a.turn + t * half);
        if (is_k) ks[c] = u * a.k_scale;
        else qs[c] = u;
    }
    const float keep = a.decay[h], low = a.decay_low[h];
    __syncthreads();
    for (int base = 0; base < d; base += kRetStepRows * rows_par) {
        if (base) request(base);
#pragma unroll
        for (int k = 0; k < kRetStepRows; k++) {
            const int n = base + k * rows_par + tr;
            if (mine && n < d) {
                const float kn = ks[n], qn = qs[n];
#pragma unroll
                for (int e = 0; e < VEC; e++) {
                    v[k][e] = kept<T>(v[k][e], keep, low, kn * x[e]);
                    y[e] = fmaf(v[k][e], qn, y[e]);
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
        for (int e = 0; e < VEC; e++) part[tr * cpb + cc + e] = y[e];
    }
    __syncthreads();
    float sq = 0.f;
    for (int i = threadIdx.x; i < ncol; i += blockDim.x) {
        float o = 0.f;
        for (int r = 0; r < rows_par; r++) o += part[r * cpb + i];
        os[i] = o;      // read back by the same thread only
        sq += o * o;
    }
    sq = block_sum(sq, red);
    if (gridDim.z > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        if (threadIdx.x == 0) squares = sq;
        cluster.sync();
        sq = 0.f;
        for (unsigned r = 0; r < cluster.num_blocks(); r++) sq += *cluster.map_shared_rank(&squares, r);
        cluster.sync();      // no CTA leaves while its sum may still be read
    }
    const float inv = 1.0f / sqrtf(sq / (float)dv + a.eps);
    for (int i = threadIdx.x; i < ncol; i += blockDim.x) {
        const long c = (long)h * dv + c0 + i;
        out[t * (long)a.H * dv + c] = from_f<T>(os[i] * inv * act_silu(to_f(row[a.g_off + c])));
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
#define GRANT_SMEM(kernel, smem)                                                                                                       \
    do {                                                                                                                               \
        static size_t granted = 46 * 1024; /* less the kernels' static shared memory */                                               \
        if ((smem) > granted) { KTB_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem))); granted = (smem); } \
    } while (0)

static bool ret_aligned(const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }
static bool ret_bad(const ktb200_retention_params* c) {
    return !c || !c->proj || !c->decay || !c->decay_low || !c->log2_decay || !c->seqs || !c->state || c->heads <= 0 || c->dim <= 0 || c->vdim <= 0 || c->rot_dims < 0 || c->rot_dims > c->dim ||
           (c->rot_dims & 1) || (c->rot_dims && !c->turn) || (c->rot_layout != kRotInterleaved && c->rot_layout != kRotHalves);
}
static Retention ret_args(const ktb200_retention_params* c) {
    return Retention{c->proj, c->proj_stride, c->q_off, c->k_off, c->v_off, c->g_off, c->heads, c->dim, c->vdim, c->rot_dims, c->rot_layout, reinterpret_cast<const float2*>(c->turn),
                     c->k_scale, c->decay, c->decay_low, c->log2_decay, c->eps, c->seqs, c->seqs_stride, c->n_seqs, c->state, c->state_stride};
}

extern "C" int ktb200_turn_table(const int* pos, const double* inv_freq, int pairs, float* turn, int n_tokens, void* stream) {
    if (!pos || !inv_freq || !turn || pairs <= 0 || !ret_aligned(turn, 8)) { set_error("turn_table: bad argument"); return KTB200_EINVAL; }
    if (n_tokens <= 0) return KTB200_OK;
    const long n = (long)n_tokens * pairs;
    turn_table_kernel<<<(unsigned)((n + 127) / 128 < 148 * 16 ? (n + 127) / 128 : 148 * 16), 128, 0, (cudaStream_t)stream>>>(pos, inv_freq, pairs, reinterpret_cast<float2*>(turn), n);
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}

extern "C" int ktb200_retention_scan(const ktb200_retention_params* c, float* o, int dtype, void* stream) {
    if (ret_bad(c) || !o || c->dim > kRetWarps * kRetRows) { set_error("retention_scan: bad argument (head size <= %d)", kRetWarps * kRetRows); return KTB200_EINVAL; }
    if (c->n_seqs <= 0) return KTB200_OK;
    const Retention a = ret_args(c);
    const int rpt = (((c->dim + kRetWarps - 1) / kRetWarps) + 3) & ~3, dp = rpt * kRetWarps;
    const size_t smem = ((size_t)2 * kRetChunk * dp + kRetChunk * 32 + (size_t)kRetChunk * kRetWarps * 32) * sizeof(float);
    const dim3 grid(c->n_seqs, c->heads, (c->vdim + 31) / 32);
#define SCAN_LAUNCH(ROWS)                                                                                        \
    SEQ_DISPATCH(dtype, {                                                                                        \
        GRANT_SMEM((retention_scan_kernel<T, ROWS>), smem);                                                      \
        retention_scan_kernel<T, ROWS><<<grid, kRetWarps * 32, smem, (cudaStream_t)stream>>>(a, o);              \
    })
    if (rpt <= 8) SCAN_LAUNCH(8);
    else if (rpt <= 16) SCAN_LAUNCH(16);
    else SCAN_LAUNCH(32);
#undef SCAN_LAUNCH
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}

extern "C" int ktb200_retention_chunk_supported(int dim, int vdim, int dtype) {
    return dtype == KTB200_TYPE_BF16 && dim > 0 && vdim > 0 && dim % 16 == 0 && vdim % 16 == 0 && dim <= 128 && vdim <= 128;
}
static long ret_tiles(int n_tokens, int n_seqs, int per) { return n_tokens / per + n_seqs; }      // (an upper bound: whole tiles and one partial per portion)
extern "C" size_t ktb200_retention_chunk_workspace(int heads, int dim, int vdim, int n_tokens, int n_seqs) {
    return (size_t)ret_tiles(n_tokens, n_seqs, kRetSpan) * heads * dim * vdim * sizeof(float) + (size_t)n_tokens * heads * dim * 4 * sizeof(__nv_bfloat16);
}

extern "C" int ktb200_retention_chunk(const ktb200_retention_params* c, void* out, int n_tokens, void* workspace, size_t workspace_bytes, int dtype, void* stream) {
    if (ret_bad(c) || !out || !ktb200_retention_chunk_supported(c->dim, c->vdim, dtype) || !workspace || !ret_aligned(workspace, 32) || !ret_aligned(c->proj, 16) || !ret_aligned(out, 4) ||
        !ret_aligned(c->state, 16) || !ret_aligned(c->turn, 16) || c->proj_stride % 8 || c->state_stride % 4 || c->q_off % 8 || c->k_off % 8 || c->v_off % 8 || c->g_off % 2 ||
        workspace_bytes < ktb200_retention_chunk_workspace(c->heads, c->dim, c->vdim, n_tokens, c->n_seqs)) {
        set_error("retention_chunk: bad argument (bf16, head sizes multiples of 16 up to 128, rows aligned to 16 bytes)");
        return KTB200_EINVAL;
    }
    if (n_tokens <= 0 || c->n_seqs <= 0) return KTB200_OK;
    const Retention a = ret_args(c);
    float* ws = (float*)workspace;
    __nv_bfloat16* q_rows = reinterpret_cast<__nv_bfloat16*>(ws + (size_t)ret_tiles(n_tokens, c->n_seqs, kRetSpan) * c->heads * c->dim * c->vdim);
    __nv_bfloat16* k_rows = q_rows + (size_t)n_tokens * c->heads * c->dim * 2;
    cudaStream_t st = (cudaStream_t)stream;
    const dim3 spans((unsigned)ret_tiles(n_tokens, c->n_seqs, kRetSpan), c->heads), chunks((unsigned)ret_tiles(n_tokens, c->n_seqs, kRetQ), c->heads);
    const size_t s1 = ((size_t)2 * kRetQ * (c->dim + 8) + (size_t)kRetQ * (c->vdim + 8)) * sizeof(__nv_bfloat16);
    GRANT_SMEM(retention_chunk_state_kernel, s1);
    retention_chunk_state_kernel<<<spans, 256, s1, st>>>(a, ws, q_rows, k_rows);
    KTB_LAUNCH_CHECK();
    retention_carry_kernel<<<dim3((c->dim * c->vdim / 8 + 127) / 128, c->heads, c->n_seqs), 128, 0, st>>>(a, ws);
    KTB_LAUNCH_CHECK();
    const size_t s3 = ret_out_smem(c->dim, c->vdim);
#define OUT_LAUNCH(DK, DV)                                                                                      \
    do {                                                                                                        \
        GRANT_SMEM((retention_chunk_out_kernel<DK, DV>), s3);                                                   \
        retention_chunk_out_kernel<DK, DV><<<chunks, 256, s3, st>>>(a, ws, q_rows, k_rows, (__nv_bfloat16*)out);                  \
    } while (0)
    if (c->dim <= 64 && c->vdim <= 64) OUT_LAUNCH(4, 4);
    else if (c->vdim <= 64) OUT_LAUNCH(8, 4);
    else OUT_LAUNCH(8, 8);
#undef OUT_LAUNCH
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}

extern "C" int ktb200_retention_step_max_vdim(void) { return kRetMaxBlocks * 256; }

extern "C" int ktb200_retention_step(const ktb200_retention_params* c, void* out, int dtype, void* stream) {
    if (ret_bad(c) || !out || c->vdim > ktb200_retention_step_max_vdim() || c->dim > 4096) { set_error("retention_step: bad argument"); return KTB200_EINVAL; }
    if (c->n_seqs <= 0) return KTB200_OK;
    const Retention a = ret_args(c);
    const int dv = c->vdim;
    const bool vec = dv % 4 == 0 && c->state_stride % 4 == 0 && ret_aligned(c->state, 16);
    // columns per CTA: up to 128, or 32 while that leaves SMs idle; at most kRetMaxBlocks column blocks per head
    int cpb = (long)c->n_seqs * c->heads < 2 * 148 ? 32 : 128;
    const int least = (dv + kRetMaxBlocks - 1) / kRetMaxBlocks;
    if (cpb < least) cpb = least;
    if (cpb > dv) cpb = dv;
    if (vec) cpb = (cpb + 3) & ~3;
    const int blocks = (dv + cpb - 1) / cpb, rows_par = 256 / (vec ? cpb / 4 : cpb);
    const size_t smem = ((size_t)2 * ((c->dim + 3) & ~3) + ((cpb + 3) & ~3) + (size_t)rows_par * cpb) * sizeof(float);
    cudaLaunchConfig_t cfg{};
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeClusterDimension;
    attr.val.clusterDim.x = 1;
    attr.val.clusterDim.y = 1;
    attr.val.clusterDim.z = blocks;
    cfg.gridDim = dim3(c->n_seqs, c->heads, blocks);
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = (cudaStream_t)stream;
    cfg.attrs = &attr;
    cfg.numAttrs = 1;
    SEQ_DISPATCH(dtype, {
        if (vec) KTB_CUDA_CHECK(cudaLaunchKernelEx(&cfg, retention_step_kernel<T, 4>, a, (T*)out, cpb));
        else KTB_CUDA_CHECK(cudaLaunchKernelEx(&cfg, retention_step_kernel<T, 1>, a, (T*)out, cpb));
    });
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}
