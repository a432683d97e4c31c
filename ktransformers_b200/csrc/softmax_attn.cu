// Soft-max attention over grouped key/value heads in a paged cache, with a partial rotation, normed queries and keys, capped
// scores, a logarithmic distance bias, a sink, a sliding-window or chunked mask, an output gate, differential pairs of maps, and values blended
// with another layer's (libktb200_seq.so).
//
//   ktb200_qkv_prep       proj rows [... q ... k ... v ...], q and k with `maps` rows of d columns per head: a causal filter of `taps` taps along time
//                         on every channel (optional); q and k turn over their first rot_dims columns (pairs of either layout, angle
//                         pos * inv_freq[i]), then (qk_norm 1) are scaled to unit rms row by row, or (qk_norm 2) divided by the rms of the WHOLE
//                         q (k) row and multiplied by a weight per column, or (qk_norm 3) scaled to unit rms row by row and multiplied by one weight row of d numbers
//                         AHEAD of the rotation; v <- (1 - t) v + t v_other with one learned t (optional), then each
//                         value head to unit rms (optional); [k | v] into the paged cache, q into q_out.
//                         ktb200_rope_norm_cache_write: the same with one map and no filter, arguments spelled out
//   ktb200_softmax_attn   o_i = sum_j softmax_j(s_ij) v_j over the keys j <= i with i - j < window (window > 0) and floor(j / chunk) ==
//                         floor(i / chunk) (chunk > 0);  s_ij = cap(scale t_h q_i.k_j) - r1_h ln(1 + r2_h (i - j)), cap(s) = c tanh(s / c),
//                         c = softcap (softcap <= 0: none), t_h, r1_h, r2_h learned numbers per query head (optional); the denominator also
//                         counts exp(sink_h) (optional); query head h reads key/value head h / (H / G).  Two maps: two such attentions per
//                         head over the same values, o = unit rms of (first - lambda second).  o times out_scale times sigmoid(gate)
//                         (optional, element by element) goes to a row of any stride.  The key range is cut into splits for few tokens on
//                         long ranges; bf16 with head sizes that are multiples of 16 up to 128: m16n8k16 tensor-core tiles.
//                         ktb200_window_softmax_attn: the plain case, arguments spelled out
//
// Storage type T (bf16 or float) for activations and cache rows; rotation, norms, scores, the cap and the soft-max are fp32
// (angles fp64).  Cache row of a token: [k G*maps*d | v G*dv]; a sequence's page table row is a ring.
#include <cuda_bf16.h>

#include "common.cuh"
#include "seq_common.cuh"
#include "mma_tile.cuh"

namespace ktb {

// ------------------------------------------------------------------------------------------------ filter, rotation, unit rms, value blend, cache write
// grid (tokens, unit blocks): a token's units are its `maps` H query rows, then its `maps` G key rows (one per head and map), then its G value
// heads; a CTA takes `units_per_cta` consecutive units, a warp per unit.  Prompt-sized batches run one CTA per token; small batches spread a
// token's units over several CTAs so that a decode step is not one warp's chain of heads.  What a CTA with query or key units needs of the
// whole token it computes itself: the rot_dims / 2 (cos, sin) pairs (fp64 angle and sincos, kept as fp32) and, for the row-wide norm, the
// sums of squares of the whole q row and the whole k row (16- / 8-byte loads where the rows allow them, one fixed order of addition).
// CONV: every channel of q, k and v first passes a causal filter along time; a unit's filtered columns sit in shared memory so that a rotated
// column finds its partner, and the CTAs of a portion's last token move the last taps - 1 inputs into the portion's state row.
constexpr int kPrepMaxPerLane = 8;      // head size <= 256
constexpr int kQkNormNone = 0, kQkNormHead = 1, kQkNormRow = 2, kQkNormHeadFirst = 3;
struct QkvPrep {
    const void* proj;
    long proj_stride;
    int q_off, k_off, v_off, Hq, Gk, Gv, d, dv, rot_dims, rot_layout;
    const double* inv_freq;
    int qk_norm;
    const void *q_w, *k_w;
    int v_unit_rms;
    float eps;
    const void* v_other;
    long v_other_stride;
    const float* blend;
    const void* conv_w;      // [Hq d + Gk d + Gv dv][taps]
    int taps;
    const int *seq_of, *seqs;
    int seqs_stride;
    float* state;
    long state_stride, conv_off;
    const int *pos, *slot, *page_table;
    int max_pages, page_size;
    void *cache, *q_out;
    int units_per_cta, vec_rows;
};
template <typename T>
__device__ __forceinline__ float sum_squares(const T* __restrict__ x, int n, bool vec) {
    float s = 0.f;
    if (vec) {
        for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
            const float4 v = load4(x + i);
            s += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = to_f(x[i]); s += v * v; }
    }
    return s;
}
template <typename T, bool CONV>
__global__ void __launch_bounds__(256) rope_norm_cache_write_kernel(const QkvPrep a) {
    __shared__ float2 turn[16 * kPrepMaxPerLane];      // (cos, sin) of the token's angles
    __shared__ float red[8], row_inv[2];
    __shared__ float filtered[CONV ? 8 : 1][CONV ? 32 * kPrepMaxPerLane : 1];
    const long t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int H = a.Hq, G = a.Gk, d = a.d, dv = a.dv;
    const int units = H + G + a.Gv, u0 = blockIdx.y * a.units_per_cta, u1 = min(units, u0 + a.units_per_cta);
    const int p = a.pos[t], half = a.rot_dims >> 1;
    const T* row = (const T*)a.proj + t * a.proj_stride;
    if (u0 < H + G) {      // this CTA has query or key heads
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            double sn, cs;
            sincos((double)p * a.inv_freq[i], &sn, &cs);
            turn[i] = make_float2((float)cs, (float)sn);
        }
        if (a.qk_norm == kQkNormRow) {      // a turn keeps x^2 + y^2 of its pair: the row's mean square is that of the un-turned columns
            const float sq = block_sum(sum_squares(row + a.q_off, H * d, a.vec_rows), red);
            const float sk = block_sum(sum_squares(row + a.k_off, G * d, a.vec_rows), red);
            if (threadIdx.x == 0) {
                row_inv[0] = 1.0f / sqrtf(sq / (float)(H * d) + a.eps);
                row_inv[1] = 1.0f / sqrtf(sk / (float)(G * d) + a.eps);
            }
        }
        __syncthreads();
    }
    const long crow = ((long)a.page_table[(long)a.slot[t] * a.max_pages + (p / a.page_size) % a.max_pages] * a.page_size + p % a.page_size) * ((long)G * d + (long)a.Gv * dv);
    const float lam = a.v_other ? a.blend[0] : 0.f;
    T* cache = (T*)a.cache;
    ConvRows<T> cv;
    bool last = false;
    if (CONV) {
        const int s = a.seq_of[t];
        const int start = a.seqs[s], len = a.seqs[a.seqs_stride + s], rd = a.seqs[2 * a.seqs_stride + s], wr = a.seqs[3 * a.seqs_stride + s];
        cv = ConvRows<T>{(const T*)a.proj + (long)start * a.proj_stride, a.proj_stride, (const T*)a.conv_w, a.taps, H * d + G * d + a.Gv * dv,
                         rd >= 0 ? a.state + (long)rd * a.state_stride + a.conv_off : nullptr, wr >= 0 ? a.state + (long)wr * a.state_stride + a.conv_off : nullptr,
                         (int)t - start};
        last = (int)t - start == len - 1 && wr >= 0;
    }
    for (int hh = u0 + warp; hh < min(u1, H + G); hh += nw) {
        const bool is_q = hh < H;
        const int col0 = is_q ? a.q_off + hh * d : a.k_off + (hh - H) * d;      // first column in proj
        const int ch0 = hh * d;                                                  // first filtered channel
        const T* src = row + col0;
        if (CONV) {
            for (int i = lane; i < d; i += 32) filtered[warp][i] = cv.value(col0 + i, ch0 + i);
            __syncwarp();
        }
        const T* first_w = a.qk_norm == kQkNormHeadFirst ? (is_q ? (const T*)a.q_w : (const T*)a.k_w) : nullptr;
        auto column = [&](int i) -> float { return CONV ? filtered[warp][i] : to_f(src[i]); };
        float r[kPrepMaxPerLane];
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < kPrepMaxPerLane; e++) {
            const int i = lane + 32 * e;
            r[e] = 0.f;
            if (i < d) {
                float v = column(i);
                const float raw = v;
                if (first_w) v *= to_f(first_w[i]);      // (the unit-rms factor is one number per row: it follows the rotation)
                if (i < a.rot_dims) {
                    const int pi = rot_partner(i, a.rot_dims, a.rot_layout);
                    float other = column(pi);
                    if (first_w) other *= to_f(first_w[pi]);
                    const bool second = a.rot_layout == kRotHalves ? i >= half : (i & 1);
                    const float2 cs = turn[a.rot_layout == kRotHalves ? (second ? i - half : i) : (i >> 1)];
                    v = second ? v * cs.x + other * cs.y : v * cs.x - other * cs.y;
                }
                r[e] = v;
                s += first_w ? raw * raw : v * v;
            }
        }
        float inv = 1.f;
        if (a.qk_norm == kQkNormHead || first_w) {
            s = warp_sum(s);
            inv = 1.0f / sqrtf(s / (float)d + a.eps);
        } else if (a.qk_norm == kQkNormRow) {
            inv = row_inv[is_q ? 0 : 1];
        }
        T* dst = is_q ? (T*)a.q_out + (t * H + hh) * d : cache + crow + (long)(hh - H) * d;
        const T* wrow = a.qk_norm == kQkNormRow ? (is_q ? (const T*)a.q_w + (long)hh * d : (const T*)a.k_w + (long)(hh - H) * d) : nullptr;
#pragma unroll
        for (int e = 0; e < kPrepMaxPerLane; e++) {
            const int i = lane + 32 * e;
            if (i < d) dst[i] = from_f<T>(wrow ? r[e] * inv * to_f(wrow[i]) : r[e] * inv);
        }
        if (CONV) {
            if (last)
                for (int i = lane; i < d; i += 32) cv.store_tail(col0 + i, ch0 + i);
            __syncwarp();
        }
    }
    // value heads: blend, mean square over the head's columns (optional), the scaled columns into the cache
    for (int hh = max(u0, H + G) + warp; hh < u1; hh += nw) {
        const int g = hh - H - G;
        const T* v = row + a.v_off + (long)g * dv;
        const T* vo = a.v_other ? (const T*)a.v_other + t * a.v_other_stride + (long)g * dv : nullptr;
        T* dst = cache + crow + (long)G * d + (long)g * dv;
        const int col0 = a.v_off + g * dv, ch0 = (H + G) * d + g * dv;
        auto column = [&](int i) -> float {
            float x = CONV ? cv.value(col0 + i, ch0 + i) : to_f(v[i]);
            if (vo) x = (1.0f - lam) * x + lam * to_f(vo[i]);
            return x;
        };
        float inv = 1.f;
        if (a.v_unit_rms) {
            float s = 0.f;
            for (int i = lane; i < dv; i += 32) {
                const float x = column(i);
                s += x * x;
            }
            inv = 1.0f / sqrtf(warp_sum(s) / (float)dv + a.eps);
        }
        for (int i = lane; i < dv; i += 32) {
            const float x = column(i);
            dst[i] = from_f<T>(a.v_unit_rms ? x * inv : x);
            if (CONV && last) cv.store_tail(col0 + i, ch0 + i);
        }
    }
}

// The same behind a filter, by column pairs: grid (tiles of `tile` consecutive tokens, unit blocks), a warp per unit walks over the tile's tokens with
// the filter's last TAPS - 1 inputs in registers, a lane owning the column pairs 2 lane + 64 e: every input is read once per tile instead of TAPS
// times, a rotated pair (interleaved layout) lies in one lane, loads and stores take two columns.  Loads of kPairBatch tokens are in flight
// together.  Without norms the maps of a head are one unit (a column turns by its place among turn_width).  Even head sizes and offsets; no row-wide norm, value blend or value norm (those take the kernel above).
constexpr int kPairTile = 16, kPairBatch = 4;
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}
__device__ __forceinline__ void store2(float* p, float x, float y) { *reinterpret_cast<float2*>(p) = make_float2(x, y); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float x, float y) { *reinterpret_cast<uint32_t*>(p) = pack_bf16(x, y); }

template <typename T, int TAPS, int PAIRS>
__global__ void __launch_bounds__(256, PAIRS > 2 ? 1 : 2) conv_rope_cache_write_kernel(const QkvPrep a, int n_tokens, int tile, int turn_width) {
    extern __shared__ __align__(16) float2 turn_s[];      // [tile][rot_dims / 2] (cos, sin)
    __shared__ int info[kPairTile][5];                    // per token: first row, tokens, row to read, row to write of its portion; cache row
    constexpr int BACK = TAPS - 1;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int H = a.Hq, G = a.Gk, d = a.d, dv = a.dv, half = a.rot_dims >> 1, C = (H + G) * d + a.Gv * dv;
    const int t0 = blockIdx.x * tile, nt = min(tile, n_tokens - t0);
    const int units = H + G + a.Gv, u0 = blockIdx.y * a.units_per_cta, u1 = min(units, u0 + a.units_per_cta);
    if (threadIdx.x < nt) {
        const int t = t0 + threadIdx.x, s = a.seq_of[t], p = a.pos[t];
#pragma unroll
        for (int k = 0; k < 4; k++) info[threadIdx.x][k] = a.seqs[k * a.seqs_stride + s];
        info[threadIdx.x][4] = a.page_table[(long)a.slot[t] * a.max_pages + (p / a.page_size) % a.max_pages] * a.page_size + p % a.page_size;
    }
    if (u0 < H + G)
        for (int i = threadIdx.x; i < nt * half; i += blockDim.x) {
            const int tt = i / half;
            double sn, cs;
            sincos((double)a.pos[t0 + tt] * a.inv_freq[i - tt * half], &sn, &cs);
            turn_s[i] = make_float2((float)cs, (float)sn);
        }
    __syncthreads();
    const T* proj = (const T*)a.proj;
    const T* cw = (const T*)a.conv_w;
    T* cache = (T*)a.cache;
    const long row_width = (long)G * d + (long)a.Gv * dv;
    for (int u = u0 + warp; u < u1; u += nw) {
        const bool is_v = u >= H + G, is_q = u < H;
        const int n = is_v ? dv : d, ch0 = is_v ? (H + G) * d + (u - H - G) * dv : u * d;
        const int col0 = is_q ? a.q_off + u * d : (is_v ? a.v_off + (u - H - G) * dv : a.k_off + (u - H) * d);
        float w[TAPS][PAIRS][2], win[BACK][PAIRS][2];
#pragma unroll
        for (int e = 0; e < PAIRS; e++) {
            const int i = 2 * lane + 64 * e;
#pragma unroll
            for (int j = 0; j < TAPS; j++) {
                w[j][e][0] = i < n ? to_f(cw[(long)(ch0 + i) * TAPS + j]) : 0.f;
                w[j][e][1] = i < n ? to_f(cw[(long)(ch0 + i + 1) * TAPS + j]) : 0.f;
            }
        }
        int at_turn[PAIRS];      // which pair of its map a lane's column pair is
#pragma unroll
        for (int e = 0; e < PAIRS; e++) at_turn[e] = ((2 * lane + 64 * e) % turn_width) >> 1;
        int cur = -1;
        for (int b = 0; b < nt; b += kPairBatch) {
            float2 in[kPairBatch][PAIRS];
#pragma unroll
            for (int k = 0; k < kPairBatch; k++)
#pragma unroll
                for (int e = 0; e < PAIRS; e++) {
                    const int i = 2 * lane + 64 * e;
                    in[k][e] = b + k < nt && i < n ? load2(proj + (long)(t0 + b + k) * a.proj_stride + col0 + i) : make_float2(0.f, 0.f);
                }
#pragma unroll
            for (int k = 0; k < kPairBatch; k++) {
                const int tt = b + k;
                if (tt >= nt) break;
                const int start = info[tt][0], len = info[tt][1], rd = info[tt][2], wr = info[tt][3], off = t0 + tt - start;
                if (start != cur) {      // another portion, or the tile's first token: fetch the inputs ahead of it
                    cur = start;
#pragma unroll
                    for (int j = 0; j < BACK; j++)
#pragma unroll
                        for (int e = 0; e < PAIRS; e++) {
                            const int i = 2 * lane + 64 * e, at = off - BACK + j;
                            float2 v = make_float2(0.f, 0.f);
                            if (i < n) {
                                if (at >= 0) v = load2(proj + (long)(start + at) * a.proj_stride + col0 + i);
                                else if (rd >= 0) {
                                    const float* st = a.state + (long)rd * a.state_stride + a.conv_off + (long)(BACK + at) * C + ch0 + i;
                                    v = make_float2(st[0], st[1]);
                                }
                            }
                            win[j][e][0] = v.x;
                            win[j][e][1] = v.y;
                        }
                }
                float y[PAIRS][2], ss = 0.f;
#pragma unroll
                for (int e = 0; e < PAIRS; e++) {
                    const int i = 2 * lane + 64 * e;
                    float x0 = 0.f, x1 = 0.f;
#pragma unroll
                    for (int j = 0; j < BACK; j++) {
                        x0 = fmaf(w[j][e][0], win[j][e][0], x0);
                        x1 = fmaf(w[j][e][1], win[j][e][1], x1);
                    }
                    x0 = fmaf(w[BACK][e][0], in[k][e].x, x0);
                    x1 = fmaf(w[BACK][e][1], in[k][e].y, x1);
#pragma unroll
                    for (int j = 0; j + 1 < BACK; j++) {
                        win[j][e][0] = win[j + 1][e][0];
                        win[j][e][1] = win[j + 1][e][1];
                    }
                    win[BACK - 1][e][0] = in[k][e].x;
                    win[BACK - 1][e][1] = in[k][e].y;
                    if (!is_v && at_turn[e] < half) {
                        const float2 cs = turn_s[tt * half + at_turn[e]];
                        const float z = x0;
                        x0 = z * cs.x - x1 * cs.y;
                        x1 = x1 * cs.x + z * cs.y;
                    }
                    y[e][0] = x0;
                    y[e][1] = x1;
                    ss += x0 * x0 + x1 * x1;
                }
                const float inv = !is_v && a.qk_norm == kQkNormHead ? 1.0f / sqrtf(warp_sum(ss) / (float)d + a.eps) : 1.0f;
                T* dst = is_q ? (T*)a.q_out + ((long)(t0 + tt) * H + u) * d : cache + (long)info[tt][4] * row_width + (is_v ? (long)G * d + (u - H - G) * dv : (long)(u - H) * d);
#pragma unroll
                for (int e = 0; e < PAIRS; e++) {
                    const int i = 2 * lane + 64 * e;
                    if (i < n) {
                        store2(dst + i, y[e][0] * inv, y[e][1] * inv);
                        if (off == len - 1 && wr >= 0) {
#pragma unroll
                            for (int j = 0; j < BACK; j++) {
                                float* st = a.state + (long)wr * a.state_stride + a.conv_off + (long)j * C + ch0 + i;
                                st[0] = win[j][e][0];
                                st[1] = win[j][e][1];
                            }
                        }
                    }
                }
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ soft-max attention, CUDA cores
// grid (tokens, G * head blocks, splits); a warp per query head (HB = blockDim / 32 heads of ONE key/value head per CTA).  Tiles of
// 32 keys in shared memory as fp32: lane = key for the scores, lane = value column for the weighted sum; running maximum and sum per
// warp.  Shared memory:  q [HB][d] | K [32][d + 1] | V [32][dv] | weights [HB][32]
constexpr int kSmTile = 32;
constexpr int kSmMaxCols = 8;      // value columns per lane: vdim <= 256
__device__ __forceinline__ float cap_score(float s, float softcap) { return softcap > 0.f ? softcap * tanhf(s / softcap) : s; }
// the first key that the query at position p sees: the start of its window, or of its chunk (chunks are counted from position 0)
__device__ __forceinline__ int first_visible(int p, int window, int chunk) {
    int lo = window > 0 ? max(0, p - window + 1) : 0;
    if (chunk > 0) lo = max(lo, p - p % chunk);
    return lo;
}

// what the attention kernels read and write; query row of a token: [head][map][d], cache row: [key/value head][map][d] keys, then [key/value head][dv] values
struct SmAttn {
    const void* q;
    int H, G, M, d, dv;
    float scale;
    const float* head_scale;
    float softcap;
    int window, chunk;
    const float *r1, *r2;      // scores lose r1[h] ln(1 + r2[h] (i - j))
    const float* sink;         // exp(sink[h]) joins the denominator
    const void* gate;          // out *= sigmoid(gate[t * gate_stride + h dv + c])
    long gate_stride;
    float out_scale;
    const float* lambda;       // M = 2: out = unit rms of (first map - lambda[0] second map)
    float rms_eps;
    const int *pos, *slot, *seqs;
    int seqs_stride, n_seqs, RH;
    const int* page_table;
    int max_pages, page_size;
    const void* cache;
    void* out;
    long out_stride;
    float* partial;            // [T][H][M][splits][dv + 2]: running maximum, sum, un-normalised weighted values
    int splits;
};
__device__ __forceinline__ float sm_sigmoid(float x) { return __fdiv_rn(1.0f, 1.0f + expf(-x)); }

template <typename T>
__global__ void __launch_bounds__(256) window_softmax_attn_kernel(const SmAttn a) {
    extern __shared__ __align__(16) float sm[];
    const int HB = blockDim.x >> 5, R = a.H / a.G, hblocks = (R + HB - 1) / HB, d = a.d, dv = a.dv, M = a.M;
    const int hb = blockIdx.y % hblocks, map = (blockIdx.y / hblocks) % M, g = blockIdx.y / (hblocks * M);
    const long t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r = hb * HB + warp, h = g * R + r;
    const bool live = r < R;
    float* qs = sm;
    float* Ks = qs + HB * d;
    float* Vs = Ks + kSmTile * (d + 1);
    float* pw = Vs + kSmTile * dv;
    const int p = a.pos[t];
    // this split's part of the visible range [lo, p], in whole tiles counted from lo
    const int lo = first_visible(p, a.window, a.chunk), n_keys = p + 1 - lo;
    const int splits = a.splits;
    const int per = ((n_keys + splits - 1) / splits + kSmTile - 1) / kSmTile * kSmTile;
    const int k_lo = lo + blockIdx.z * per, k_hi = min(p + 1, k_lo + per);
    const T* cache = (const T*)a.cache;
    float acc[kSmMaxCols];
#pragma unroll
    for (int c = 0; c < kSmMaxCols; c++) acc[c] = 0.f;
    float m = -INFINITY, l = 0.f;
    if (k_lo < k_hi) {
        const float r1 = live && a.r1 ? a.r1[h] : 0.f, r2 = live && a.r1 ? a.r2[h] : 0.f;
        if (live) {
            const float sc = a.head_scale ? a.scale * a.head_scale[h] : a.scale;
            for (int i = lane; i < d; i += 32) qs[warp * d + i] = to_f(((const T*)a.q)[((t * a.H + h) * M + map) * d + i]) * sc;
        }
        const int* pt = a.page_table + (long)a.slot[t] * a.max_pages;
        const long cw = (long)a.G * (M * d + dv);
        for (int j0 = k_lo; j0 < k_hi; j0 += kSmTile) {
            __syncthreads();
            const int nk = min(kSmTile, k_hi - j0);
            for (int i = threadIdx.x; i < nk * d; i += blockDim.x) {
                const int j = i / d, c = i - j * d, kp = j0 + j;
                Ks[j * (d + 1) + c] = to_f(cache[((long)pt[(kp / a.page_size) % a.max_pages] * a.page_size + kp % a.page_size) * cw + (long)(g * M + map) * d + c]);
            }
            for (int i = threadIdx.x; i < nk * dv; i += blockDim.x) {
                const int j = i / dv, c = i - j * dv, kp = j0 + j;
                Vs[j * dv + c] = to_f(cache[((long)pt[(kp / a.page_size) % a.max_pages] * a.page_size + kp % a.page_size) * cw + (long)a.G * M * d + (long)g * dv + c]);
            }
            __syncthreads();
            if (!live) continue;
            float s = -INFINITY;
            if (lane < nk) {
                float q_k = 0.f;
                const float* kr = Ks + lane * (d + 1);
                const float* qr = qs + warp * d;
                for (int i = 0; i < d; i++) q_k = fmaf(qr[i], kr[i], q_k);
                s = cap_score(q_k, a.softcap);
                if (a.r1) s -= r1 * log1pf(r2 * (float)(p - (j0 + lane)));
            }
            const float mn = fmaxf(m, warp_max(s));      // every tile holds at least one key, so mn is finite
            const float corr = expf(m - mn);
            const float pj = expf(s - mn);
            l = l * corr + warp_sum(pj);
            m = mn;
            pw[warp * kSmTile + lane] = pj;
            __syncwarp();
#pragma unroll
            for (int c = 0; c < kSmMaxCols; c++) acc[c] *= corr;
            for (int j = 0; j < nk; j++) {
                const float wj = pw[warp * kSmTile + j];
#pragma unroll
                for (int c = 0; c < kSmMaxCols; c++)
                    if (lane + 32 * c < dv) acc[c] = fmaf(wj, Vs[j * dv + lane + 32 * c], acc[c]);
            }
            __syncwarp();
        }
    }
    if (!live) return;
    if (a.partial) {
        float* o = a.partial + (((t * a.H + h) * M + map) * splits + blockIdx.z) * (dv + 2);
        if (lane == 0) { o[0] = m; o[1] = l; }
#pragma unroll
        for (int c = 0; c < kSmMaxCols; c++)
            if (lane + 32 * c < dv) o[2 + lane + 32 * c] = acc[c];
    } else {      // (one map, one split)
        float inv = 1.0f;
        if (a.sink) {
            const float sk = a.sink[h], mn = fmaxf(m, sk), corr = expf(m - mn);
            inv = corr / (l * corr + expf(sk - mn));
        } else {
            inv = 1.0f / l;
        }
        inv *= a.out_scale;
        const T* gate = (const T*)a.gate + t * a.gate_stride + (long)h * dv;
        T* out = (T*)a.out + t * a.out_stride + (long)h * dv;
#pragma unroll
        for (int c = 0; c < kSmMaxCols; c++) {
            const int i = lane + 32 * c;
            if (i < dv) out[i] = from_f<T>(a.gate ? acc[c] * inv * sm_sigmoid(to_f(gate[i])) : acc[c] * inv);
        }
    }
}

// ------------------------------------------------------------------------------------------------ soft-max attention, tensor cores (bf16)
// A CTA of ROWS / 16 warps owns a tile of ROWS rows = (token, query head) pairs of ONE sequence portion and ONE key/value head: `RH`
// query heads of the group for each of ROWS / RH consecutive tokens (prompt portions fill the rows with tokens, decode steps with the
// group's heads, so grouped heads share every key tile).  Keys run in tiles of KEYS through a two-stage cp.async ring of [k | v]
// rows gathered through the page table, from the first key that the tile's earliest token still sees to its last token's own;
// S = Q K^T and O += P V are m16n8k16 bf16 MMAs with fp32 accumulators; scale, cap, window and causal masks, running maximum and
// sum in fp32 registers (a row's maximum over the four threads that hold it); the weights go to the second product as bf16.
// grid (tile bound, G * head blocks, splits); tiles are found from the per-sequence rows `seqs`.  Held to 128 registers (a few bytes of
// spills at head size 128) so that four CTAs share an SM: decode-shaped launches are bound by the copies in flight per SM.
constexpr int kMmaRows = 64, kMmaKeys = 32, kMmaPad = 8;
__device__ __forceinline__ float cap_score_fast(float s, float two_over_cap, float softcap) {
    // c tanh(s / c) as c (1 - 2 / (exp(2 s / c) + 1)), c = softcap: absolute error of a few 1e-7 of the cap
    return softcap * (1.0f - __fdividef(2.0f, __expf(s * two_over_cap) + 1.0f));
}

template <int D16MAX, int DV16MAX, int MAPS, bool BIAS>
__global__ void __launch_bounds__(kMmaRows * 2, 4) window_softmax_attn_mma_kernel(const SmAttn a) {
    constexpr int ROWS = kMmaRows / MAPS, KEYS = kMmaKeys, WPM = 4 / MAPS;      // (token, head) rows; warps per map
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ int tile_info[3];
    const int tid = threadIdx.x, lane = tid & 31, warp = MAPS == 1 ? tid >> 5 : (tid >> 5) % WPM, map = MAPS == 1 ? 0 : (tid >> 5) / WPM, gq = lane >> 2, tq = lane & 3;
    const __nv_bfloat16* __restrict__ q = (const __nv_bfloat16*)a.q;
    const __nv_bfloat16* __restrict__ cache = (const __nv_bfloat16*)a.cache;
    const int H = a.H, G = a.G, d = a.d, dv = a.dv, RH = a.RH, window = a.window, chunk = a.chunk, max_pages = a.max_pages, page_size = a.page_size;
    const int *pos = a.pos, *seqs = a.seqs, seqs_stride = a.seqs_stride, n_seqs = a.n_seqs;
    const float scale = a.scale, softcap = a.softcap;
    const int TOKS = ROWS / RH;
    if (tid == 0) {      // which sequence portion and which of its tokens this tile covers
        int b = blockIdx.x, found = -1, off = 0, len = 0;
        for (int s = 0; s < n_seqs; s++) {
            len = seqs[seqs_stride + s];
            const int nt = (len + TOKS - 1) / TOKS;
            if (b < nt) { found = s; off = b * TOKS; break; }
            b -= nt;
        }
        tile_info[0] = found;
        tile_info[1] = found >= 0 ? seqs[found] + off : 0;
        tile_info[2] = found >= 0 ? min(TOKS, len - off) : 0;
    }
    __syncthreads();
    if (tile_info[0] < 0) return;
    const int tok0 = tile_info[1], ntok = tile_info[2];
    const int R = H / G, hblocks = R / RH;
    const int g = blockIdx.y / hblocks, h0 = g * R + (blockIdx.y % hblocks) * RH;
    const int d16 = d >> 4, dv16 = dv >> 4, ldk = MAPS * d + kMmaPad, ldv = dv + kMmaPad;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* Ks = Qs + ROWS * ldk;                     // [2][KEYS][ldk]
    __nv_bfloat16* Vs = Ks + 2 * KEYS * ldk;                 // [2][KEYS][ldv]
    const int pos0 = pos[tok0], max_pos = pos0 + ntok - 1;
    // the tile's key range [lo, max_pos], cut into this split's part in whole key tiles counted from lo
    const int lo = first_visible(pos0, window, chunk);
    const int splits = a.splits, n_keys = max_pos + 1 - lo;
    const int per = ((n_keys + splits - 1) / splits + KEYS - 1) / KEYS * KEYS;
    const int k_lo = lo + blockIdx.z * per, k_hi = min(max_pos + 1, k_lo + per);
    // this thread's two rows of the warp's 16
    const int rA = warp * 16 + gq, rB = rA + 8;
    const int tokA = rA / RH, tokB = rB / RH, hA = h0 + rA % RH, hB = h0 + rB % RH;
    const bool vA = tokA < ntok, vB = tokB < ntok;
    const int pA = pos0 + tokA, pB = pos0 + tokB;
    const int fA = first_visible(pA, window, chunk), fB = first_visible(pB, window, chunk);
    const float scA = a.head_scale ? scale * a.head_scale[hA] : scale, scB = a.head_scale ? scale * a.head_scale[hB] : scale;
    // distance bias: r1 ln(1 + r2 n) = (r1 ln 2) log2(1 + r2 n); positions as floats (exact below 2^24)
    const float b1A = BIAS ? a.r1[hA] * 0.6931471805599453f : 0.f, b1B = BIAS ? a.r1[hB] * 0.6931471805599453f : 0.f;
    const float b2A = BIAS ? a.r2[hA] : 0.f, b2B = BIAS ? a.r2[hB] : 0.f;
    const bool warp_live = (warp * 16) / RH < ntok;
    const int warp_max_pos = pos0 + min(ntok - 1, (warp * 16 + 15) / RH), warp_min_pos = pos0 + (warp * 16) / RH;
    const int warp_first_key = first_visible(warp_min_pos, window, chunk);      // no row of this warp sees a key before this one
    const int warp_last_first = first_visible(warp_max_pos, window, chunk);    // every row of this warp sees the keys from here to its own
    const float two_over_cap = softcap > 0.f ? 2.0f / softcap : 0.f;
    float O[2 * DV16MAX][4];
#pragma unroll
    for (int n = 0; n < 2 * DV16MAX; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) O[n][e] = 0.f;
    float mA = -INFINITY, mB = -INFINITY, lA = 0.f, lB = 0.f;
    if (k_lo < k_hi) {
        const int* pt = a.page_table + (long)a.slot[tok0] * max_pages;
        const long cw = (long)G * (MAPS * d + dv);
        const int kc = (MAPS * d) >> 3, vc = dv >> 3;      // 16-byte chunks per row
        for (int i = tid; i < ROWS * kc; i += blockDim.x) {
            const int r = i / kc, c = i - r * kc, tk = r / RH;
            const bool ok = tk < ntok;
            cp_async16(Qs + r * ldk + c * 8, ok ? q + ((long)(tok0 + tk) * H + h0 + r % RH) * (MAPS * d) + c * 8 : q, ok);
        }
        // TPR neighbouring threads copy key row r of a tile: one page-table lookup per thread and tile, made a tile ahead of its copies
        constexpr int TPR = kMmaRows * 2 / KEYS;
        const int lrow = tid / TPR, lpar = tid % TPR;
        auto row_base = [&](int kp) -> long {
            return kp < k_hi ? ((long)pt[(kp / page_size) % max_pages] * page_size + kp % page_size) * cw : -1;
        };
        auto load_tile = [&](int stage, long base) {
            __nv_bfloat16* kd = Ks + stage * KEYS * ldk + lrow * ldk;
            __nv_bfloat16* vd = Vs + stage * KEYS * ldv + lrow * ldv;
            const bool ok = base >= 0;
            const __nv_bfloat16* ksrc = ok ? cache + base + (long)g * (MAPS * d) : cache;
            const __nv_bfloat16* vsrc = ok ? cache + base + (long)G * (MAPS * d) + (long)g * dv : cache;
            for (int c = lpar; c < kc; c += TPR) cp_async16(kd + c * 8, ok ? ksrc + c * 8 : cache, ok);
            for (int c = lpar; c < vc; c += TPR) cp_async16(vd + c * 8, ok ? vsrc + c * 8 : cache, ok);
        };
        load_tile(0, row_base(k_lo + lrow));
        long next_base = row_base(k_lo + KEYS + lrow);
        int stage = 0;
        for (int j0 = k_lo; j0 < k_hi; j0 += KEYS, stage ^= 1) {
            cp_async_wait_all();
            __syncthreads();      // this tile has landed, and every warp is done with the other stage
            if (j0 + KEYS < k_hi) {
                load_tile(stage ^ 1, next_base);
                next_base = row_base(j0 + 2 * KEYS + lrow);
            }
            if (!warp_live || j0 > warp_max_pos || j0 + KEYS <= warp_first_key) continue;
            const __nv_bfloat16* kt = Ks + stage * KEYS * ldk + map * d;
            const __nv_bfloat16* vt = Vs + stage * KEYS * ldv;
            float S[KEYS / 8][4];
#pragma unroll
            for (int n = 0; n < KEYS / 8; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) S[n][e] = 0.f;
#pragma unroll
            for (int kk = 0; kk < D16MAX; kk++) {
                if (kk < d16) {
                    uint32_t qa[4];
                    ldmatrix_x4(qa, Qs + (warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldk + map * d + kk * 16 + 8 * (lane >> 4));
#pragma unroll
                    for (int np = 0; np < KEYS / 16; np++) {      // two key n-tiles per ldmatrix
                        uint32_t b[4];
                        ldmatrix_x4(b, kt + (np * 16 + (lane & 7) + 8 * (lane >> 4)) * ldk + kk * 16 + 8 * ((lane >> 3) & 1));
                        mma_bf16_16816(S[2 * np], qa, b[0], b[1]);
                        mma_bf16_16816(S[2 * np + 1], qa, b[2], b[3]);
                    }
                }
            }
            // nothing to mask: all 16 rows carry tokens, and every key of the tile lies at or before the earliest of them, inside the
            // window or chunk of the latest and inside this split
            const bool plain = (warp * 16 + 15) / RH < ntok && j0 + KEYS - 1 <= warp_min_pos && j0 >= warp_last_first && j0 + KEYS <= k_hi;
            float tmA = -INFINITY, tmB = -INFINITY;
            const float key0 = BIAS ? (float)(j0 + 2 * tq) : 0.f;
#pragma unroll
            for (int n = 0; n < KEYS / 8; n++) {
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    float s = S[n][e] * (e < 2 ? scA : scB);
                    if (softcap > 0.f) s = cap_score_fast(s, two_over_cap, softcap);
                    if (BIAS) {
                        const float n_back = (e < 2 ? (float)pA : (float)pB) - (key0 + (float)(n * 8 + (e & 1)));
                        s = fmaf(-(e < 2 ? b1A : b1B), __log2f(fmaf(e < 2 ? b2A : b2B, n_back, 1.0f)), s);      // (masked below where n_back < 0)
                    }
                    if (!plain) {
                        const int key = j0 + n * 8 + 2 * tq + (e & 1);
                        const bool second = e >= 2;
                        const bool ok = (second ? vB : vA) && key <= (second ? pB : pA) && key >= (second ? fB : fA) && key < k_hi;
                        if (!ok) s = -INFINITY;
                    }
                    S[n][e] = s;
                    if (e < 2) tmA = fmaxf(tmA, s);
                    else tmB = fmaxf(tmB, s);
                }
            }
            tmA = fmaxf(tmA, __shfl_xor_sync(0xffffffffu, tmA, 1));
            tmA = fmaxf(tmA, __shfl_xor_sync(0xffffffffu, tmA, 2));
            tmB = fmaxf(tmB, __shfl_xor_sync(0xffffffffu, tmB, 1));
            tmB = fmaxf(tmB, __shfl_xor_sync(0xffffffffu, tmB, 2));
            const float nA = fmaxf(mA, tmA), nB = fmaxf(mB, tmB);
            const float uA = nA == -INFINITY ? 0.f : nA, uB = nB == -INFINITY ? 0.f : nB;      // a row that has seen no key yet keeps weights of zero
            const float cA = __expf(mA - uA), cB = __expf(mB - uB);
            mA = nA;
            mB = nB;
            float sA = 0.f, sB = 0.f;
#pragma unroll
            for (int n = 0; n < KEYS / 8; n++) {
                S[n][0] = __expf(S[n][0] - uA);
                S[n][1] = __expf(S[n][1] - uA);
                S[n][2] = __expf(S[n][2] - uB);
                S[n][3] = __expf(S[n][3] - uB);
                sA += S[n][0] + S[n][1];
                sB += S[n][2] + S[n][3];
            }
            lA = lA * cA + sA;
            lB = lB * cB + sB;
#pragma unroll
            for (int n = 0; n < 2 * DV16MAX; n++) {
                O[n][0] *= cA;
                O[n][1] *= cA;
                O[n][2] *= cB;
                O[n][3] *= cB;
            }
#pragma unroll
            for (int kk = 0; kk < KEYS / 16; kk++) {      // 16 keys per step
                uint32_t pa[4] = {pack_bf16(S[2 * kk][0], S[2 * kk][1]), pack_bf16(S[2 * kk][2], S[2 * kk][3]), pack_bf16(S[2 * kk + 1][0], S[2 * kk + 1][1]),
                                 pack_bf16(S[2 * kk + 1][2], S[2 * kk + 1][3])};
#pragma unroll
                for (int vp = 0; vp < DV16MAX; vp++) {
                    if (vp < dv16) {
                        uint32_t b[4];
                        ldmatrix_x4_trans(b, vt + (kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldv + vp * 16 + 8 * (lane >> 4));
                        mma_bf16_16816(O[2 * vp], pa, b[0], b[1]);
                        mma_bf16_16816(O[2 * vp + 1], pa, b[2], b[3]);
                    }
                }
            }
        }
        cp_async_wait_all();
    }
    lA += __shfl_xor_sync(0xffffffffu, lA, 1);
    lA += __shfl_xor_sync(0xffffffffu, lA, 2);
    lB += __shfl_xor_sync(0xffffffffu, lB, 1);
    lB += __shfl_xor_sync(0xffffffffu, lB, 2);
    if (a.partial) {
        float* oA = a.partial + ((((long)(tok0 + tokA) * H + hA) * MAPS + map) * splits + blockIdx.z) * (dv + 2);
        float* oB = a.partial + ((((long)(tok0 + tokB) * H + hB) * MAPS + map) * splits + blockIdx.z) * (dv + 2);
        if (tq == 0) {
            if (vA) { oA[0] = mA; oA[1] = lA; }
            if (vB) { oB[0] = mB; oB[1] = lB; }
        }
#pragma unroll
        for (int n = 0; n < 2 * DV16MAX; n++) {
            const int col = n * 8 + 2 * tq;
            if (col < dv) {
                if (vA) *reinterpret_cast<float2*>(oA + 2 + col) = make_float2(O[n][0], O[n][1]);
                if (vB) *reinterpret_cast<float2*>(oB + 2 + col) = make_float2(O[n][2], O[n][3]);
            }
        }
        return;
    }
    float iA = vA ? 1.0f / lA : 0.f, iB = vB ? 1.0f / lB : 0.f;
    if (a.sink) {
        if (vA) { const float mn = fmaxf(mA, a.sink[hA]), c = __expf(mA - mn); iA = c / (lA * c + __expf(a.sink[hA] - mn)); }
        if (vB) { const float mn = fmaxf(mB, a.sink[hB]), c = __expf(mB - mn); iB = c / (lB * c + __expf(a.sink[hB] - mn)); }
    }
    if (MAPS == 2) {      // the second map's warps leave lambda a2 in shared memory, the first map's take it off their rows and norm the difference
        float* other = reinterpret_cast<float*>(smem_raw);      // [ROWS][dv + 8] over the tiles, which every warp is done with
        const int ldo = dv + 8;
        const float lam = a.lambda[0];
        __syncthreads();
        if (map == 1) {
#pragma unroll
            for (int n = 0; n < 2 * DV16MAX; n++) {
                const int col = n * 8 + 2 * tq;
                if (col < dv) {
                    *reinterpret_cast<float2*>(other + rA * ldo + col) = make_float2(O[n][0] * iA * lam, O[n][1] * iA * lam);
                    *reinterpret_cast<float2*>(other + rB * ldo + col) = make_float2(O[n][2] * iB * lam, O[n][3] * iB * lam);
                }
            }
        }
        __syncthreads();
        if (map == 1) return;
        float qA = 0.f, qB = 0.f;
#pragma unroll
        for (int n = 0; n < 2 * DV16MAX; n++) {
            const int col = n * 8 + 2 * tq;
            if (col < dv) {
                const float2 u = *reinterpret_cast<const float2*>(other + rA * ldo + col), w = *reinterpret_cast<const float2*>(other + rB * ldo + col);
                O[n][0] = O[n][0] * iA - u.x;
                O[n][1] = O[n][1] * iA - u.y;
                O[n][2] = O[n][2] * iB - w.x;
                O[n][3] = O[n][3] * iB - w.y;
                qA += O[n][0] * O[n][0] + O[n][1] * O[n][1];
                qB += O[n][2] * O[n][2] + O[n][3] * O[n][3];
            }
        }
        qA += __shfl_xor_sync(0xffffffffu, qA, 1);
        qA += __shfl_xor_sync(0xffffffffu, qA, 2);
        qB += __shfl_xor_sync(0xffffffffu, qB, 1);
        qB += __shfl_xor_sync(0xffffffffu, qB, 2);
        iA = 1.0f / sqrtf(qA / (float)dv + a.rms_eps);
        iB = 1.0f / sqrtf(qB / (float)dv + a.rms_eps);
    }
    iA *= a.out_scale;
    iB *= a.out_scale;
    __nv_bfloat16* out = (__nv_bfloat16*)a.out;
    const __nv_bfloat16* gate = (const __nv_bfloat16*)a.gate;
#pragma unroll
    for (int n = 0; n < 2 * DV16MAX; n++) {
        const int col = n * 8 + 2 * tq;
        if (col < dv) {
            float x[4] = {O[n][0] * iA, O[n][1] * iA, O[n][2] * iB, O[n][3] * iB};
            if (gate) {
                if (vA) {
                    const uint32_t u = *reinterpret_cast<const uint32_t*>(gate + (long)(tok0 + tokA) * a.gate_stride + hA * dv + col);
                    x[0] *= sm_sigmoid(__uint_as_float(u << 16));
                    x[1] *= sm_sigmoid(__uint_as_float(u & 0xffff0000u));
                }
                if (vB) {
                    const uint32_t u = *reinterpret_cast<const uint32_t*>(gate + (long)(tok0 + tokB) * a.gate_stride + hB * dv + col);
                    x[2] *= sm_sigmoid(__uint_as_float(u << 16));
                    x[3] *= sm_sigmoid(__uint_as_float(u & 0xffff0000u));
                }
            }
            if (vA) *reinterpret_cast<uint32_t*>(out + (long)(tok0 + tokA) * a.out_stride + hA * dv + col) = pack_bf16(x[0], x[1]);
            if (vB) *reinterpret_cast<uint32_t*>(out + (long)(tok0 + tokB) * a.out_stride + hB * dv + col) = pack_bf16(x[2], x[3]);
        }
    }
}

// one CTA of 128 threads per map for each (token, head): the parts' weights exp(m_s - m) / l once in shared memory (parts without a key have
// m = -inf and weigh nothing; the sink joins l), then the columns in parallel, parts in order; two maps are combined and the row normed here
constexpr int kMergeMaxSplits = 128;
template <typename T, int MAPS>
__global__ void __launch_bounds__(128 * MAPS) softmax_merge_kernel(const SmAttn a) {
    __shared__ float wgt_s[MAPS][kMergeMaxSplits];
    __shared__ float red_s[MAPS][4];
    __shared__ float second[MAPS == 2 ? 256 : 1];
    const long row = blockIdx.x, t = row / a.H;
    const int h = (int)(row - t * a.H), splits = a.splits, dv = a.dv;
    const int map = MAPS == 1 ? 0 : threadIdx.x >> 7, tid = threadIdx.x & 127, lane = tid & 31, warp = tid >> 5;
    float *wgt = wgt_s[map], *red = red_s[map];
    float acc[2] = {0.f, 0.f};      // columns tid and tid + 128
    const float* part = a.partial + (row * MAPS + map) * splits * (dv + 2);
    const float ms = tid < splits ? part[(long)tid * (dv + 2)] : -INFINITY;
    const float ls = tid < splits ? part[(long)tid * (dv + 2) + 1] : 0.f;
    float m = warp_max(ms);
    if (lane == 0) red[warp] = m;
    __syncthreads();
    m = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    if (a.sink) m = fmaxf(m, a.sink[h]);
    __syncthreads();
    const float e = ms > -INFINITY ? expf(ms - m) : 0.f;
    float l = warp_sum(ls * e);
    if (lane == 0) red[warp] = l;
    __syncthreads();
    l = (red[0] + red[1]) + (red[2] + red[3]);
    if (a.sink) l += expf(a.sink[h] - m);
    if (tid < splits) wgt[tid] = e / l;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 2; k++) {
        const int c = tid + 128 * k;
        if (c < dv) {
#pragma unroll 8
            for (int s = 0; s < splits; s++) acc[k] = fmaf(wgt[s], part[(long)s * (dv + 2) + 2 + c], acc[k]);
        }
    }
    float inv = a.out_scale;
    if (MAPS == 2) {
        const float lam = a.lambda[0];
        if (map == 1) {
#pragma unroll
            for (int k = 0; k < 2; k++)
                if (tid + 128 * k < dv) second[tid + 128 * k] = lam * acc[k];
        }
        __syncthreads();
        if (map == 0) {
#pragma unroll
            for (int k = 0; k < 2; k++)
                if (tid + 128 * k < dv) acc[k] -= second[tid + 128 * k];
            const float ss = warp_sum(acc[0] * acc[0] + acc[1] * acc[1]);
            if (lane == 0) red[warp] = ss;
        }
        __syncthreads();
        if (map == 1) return;
        inv *= 1.0f / sqrtf(((red[0] + red[1]) + (red[2] + red[3])) / (float)dv + a.rms_eps);
    }
    const T* gate = (const T*)a.gate + t * a.gate_stride + (long)h * dv;
    T* out = (T*)a.out + t * a.out_stride + (long)h * dv;
#pragma unroll
    for (int k = 0; k < 2; k++) {
        const int c = tid + 128 * k;
        if (c < dv) out[c] = from_f<T>(a.gate ? acc[k] * inv * sm_sigmoid(to_f(gate[c])) : acc[k] * inv);
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

extern "C" int ktb200_qkv_prep(const ktb200_qkv_prep_params* c, int n_tokens, int dtype, void* stream) {
    if (!c || !c->proj || !c->pos || !c->slot || !c->page_table || !c->cache || !c->q_out || c->heads <= 0 || c->kv_heads <= 0 || c->heads % c->kv_heads || c->maps < 1 ||
        c->dim <= 0 || c->dim > 32 * kPrepMaxPerLane || c->vdim <= 0 || c->rot_dims < 0 || c->rot_dims > c->dim || (c->rot_dims & 1) || (c->rot_dims && !c->inv_freq) ||
        (c->rot_layout != kRotInterleaved && c->rot_layout != kRotHalves) || (c->v_other && !c->blend) || c->qk_norm < kQkNormNone || c->qk_norm > kQkNormHeadFirst || (c->qk_norm == kQkNormHeadFirst && (!c->q_weight || !c->k_weight)) ||
        (c->qk_norm == kQkNormRow && (!c->q_weight || !c->k_weight || c->conv_w)) || c->page_size <= 0 || c->max_pages <= 0) {
        set_error("qkv_prep: bad argument (head size <= %d; no row-wide norm behind a filter)", 32 * kPrepMaxPerLane);
        return KTB200_EINVAL;
    }
    if (c->conv_w && (c->taps < 1 || !c->seq_of || !c->seqs || (c->taps > 1 && !c->state))) { set_error("qkv_prep: the filter needs its portions and state rows"); return KTB200_EINVAL; }
    if (n_tokens <= 0) return KTB200_OK;
    const int Hq = c->heads * c->maps, Gk = c->kv_heads * c->maps;
    // unit blocks per token: as many as keep about a wave of CTAs (148 SMs x 8) busy, eight units (one per warp) at least
    const int units = Hq + Gk + c->kv_heads, max_y = (units + 7) / 8;
    int want_y = 1184 / n_tokens;
    want_y = want_y < 1 ? 1 : (want_y > max_y ? max_y : want_y);
    const int upc = ((units + want_y - 1) / want_y + 7) / 8 * 8, grid_y = (units + upc - 1) / upc;
    const size_t esz = dtype == KTB200_TYPE_BF16 ? 2 : 4;
    const int vec_rows = c->q_off % 4 == 0 && c->k_off % 4 == 0 && (Hq * c->dim) % 4 == 0 && (Gk * c->dim) % 4 == 0 && c->proj_stride % 4 == 0 &&
                         (reinterpret_cast<uintptr_t>(c->proj) & (4 * esz - 1)) == 0;
    const QkvPrep a{c->proj, c->proj_stride, c->q_off, c->k_off, c->v_off, Hq, Gk, c->kv_heads, c->dim, c->vdim, c->rot_dims, c->rot_layout, c->inv_freq, c->qk_norm, c->q_weight,
                    c->k_weight, c->v_unit_rms, c->eps, c->v_other, c->v_other_stride, c->blend, c->conv_w, c->taps, c->seq_of, c->seqs, c->seqs_stride, c->state,
                    c->state_stride, c->conv_off, c->pos, c->slot, c->page_table, c->max_pages, c->page_size, c->cache, c->q_out, upc, vec_rows};
    const size_t two = 2 * esz;
    auto even = [&](const void* p) { return (reinterpret_cast<uintptr_t>(p) & (two - 1)) == 0; };
    const bool pairs = c->conv_w && c->taps >= 2 && c->taps <= 4 && c->dim % 2 == 0 && c->vdim % 2 == 0 && c->vdim <= 32 * kPrepMaxPerLane && c->q_off % 2 == 0 && c->k_off % 2 == 0 &&
                       c->v_off % 2 == 0 && c->proj_stride % 2 == 0 && even(c->proj) && even(c->q_out) && even(c->cache) && c->qk_norm != kQkNormRow && c->qk_norm != kQkNormHeadFirst && !c->v_other && !c->v_unit_rms &&
                       (c->rot_dims == 0 || c->rot_layout == kRotInterleaved);
    if (pairs) {      // tiles of 16 tokens once there are enough tokens to fill the SMs; unit blocks as above
        const int tile = n_tokens >= 512 ? kPairTile : (n_tokens >= 64 ? 4 : 1), tiles = (n_tokens + tile - 1) / tile;
        int y = (1184 + tiles - 1) / tiles;
        y = y > max_y ? max_y : y;
        QkvPrep b = a;
        int n_units = units;
        if (c->maps > 1 && c->qk_norm == kQkNormNone && c->dim * c->maps <= 32 * kPrepMaxPerLane) {
            b.Hq = c->heads; b.Gk = c->kv_heads; b.d = c->dim * c->maps;
            n_units = c->heads + 2 * c->kv_heads;
        }
        b.units_per_cta = ((n_units + y - 1) / y + 7) / 8 * 8;
        const dim3 grid(tiles, (n_units + b.units_per_cta - 1) / b.units_per_cta);
        const size_t smem = (size_t)tile * (c->rot_dims / 2) * sizeof(float2);
        const int widest = b.d > c->vdim ? b.d : c->vdim;
#define PAIR_LAUNCH(TAPS, PAIRS) conv_rope_cache_write_kernel<T, TAPS, PAIRS><<<grid, 256, smem, (cudaStream_t)stream>>>(b, n_tokens, tile, c->dim)
#define PAIR_SIZES(TAPS)                               \
    do {                                               \
        if (widest <= 64) PAIR_LAUNCH(TAPS, 1);        \
        else if (widest <= 128) PAIR_LAUNCH(TAPS, 2);  \
        else PAIR_LAUNCH(TAPS, 4);                     \
    } while (0)
        SEQ_DISPATCH(dtype, {
            if (c->taps == 2) PAIR_SIZES(2);
            else if (c->taps == 3) PAIR_SIZES(3);
            else PAIR_SIZES(4);
        });
#undef PAIR_SIZES
#undef PAIR_LAUNCH
        KTB_LAUNCH_CHECK();
        return KTB200_OK;
    }
    SEQ_DISPATCH(dtype, {
        if (c->conv_w) rope_norm_cache_write_kernel<T, true><<<dim3(n_tokens, grid_y), 256, 0, (cudaStream_t)stream>>>(a);
        else rope_norm_cache_write_kernel<T, false><<<dim3(n_tokens, grid_y), 256, 0, (cudaStream_t)stream>>>(a);
    });
    KTB_LAUNCH_CHECK();
    return KTB200_OK;
}

extern "C" int ktb200_rope_norm_cache_write(const void* proj, long proj_stride, int q_off, int k_off, int v_off, int heads, int kv_heads, int dim, int vdim, int rot_dims,
                                            int rot_layout, const double* inv_freq, int qk_norm, const void* q_weight, const void* k_weight, int v_unit_rms, float eps,
                                            const void* v_other, long v_other_stride, const float* blend, const int* pos, const int* slot, const int* page_table, int max_pages, int page_size, void* cache, void* q_out, int n_tokens,
                                            int dtype, void* stream) {
    ktb200_qkv_prep_params c{};
    c.proj = proj; c.proj_stride = proj_stride; c.q_off = q_off; c.k_off = k_off; c.v_off = v_off; c.heads = heads; c.kv_heads = kv_heads; c.maps = 1; c.dim = dim; c.vdim = vdim;
    c.rot_dims = rot_dims; c.rot_layout = rot_layout; c.inv_freq = inv_freq; c.qk_norm = qk_norm; c.q_weight = q_weight; c.k_weight = k_weight; c.v_unit_rms = v_unit_rms; c.eps = eps;
    c.v_other = v_other; c.v_other_stride = v_other_stride; c.blend = blend; c.pos = pos; c.slot = slot; c.page_table = page_table; c.max_pages = max_pages; c.page_size = page_size;
    c.cache = cache; c.q_out = q_out;
    return ktb200_qkv_prep(&c, n_tokens, dtype, stream);
}

/* fp32 workspace of an attention call: whenever the key range is cut, and for several maps outside the tensor-core tiles */
extern "C" size_t ktb200_softmax_attn_workspace(int n_tokens, int heads, int maps, int vdim, int splits, int tensor_cores) {
    return splits > 1 || (maps > 1 && !tensor_cores) ? (size_t)n_tokens * heads * maps * splits * (vdim + 2) * sizeof(float) : 0;
}
extern "C" size_t ktb200_window_softmax_attn_workspace(int n_tokens, int heads, int vdim, int splits) {
    return ktb200_softmax_attn_workspace(n_tokens, heads, 1, vdim, splits, 1);
}

/* whether the attention call runs tensor-core tiles for these sizes (bf16, head sizes multiples of 16 up to 128, and `seqs` given), and an
 * upper bound of its row tiles per key/value head (for choosing splits) */
extern "C" int ktb200_softmax_attn_uses_tensor_cores(int heads, int kv_heads, int maps, int dim, int vdim, int dtype) {
    return dtype == KTB200_TYPE_BF16 && kv_heads > 0 && heads % kv_heads == 0 && (maps == 1 || maps == 2) && dim % 16 == 0 && vdim % 16 == 0 && dim <= 128 && vdim <= 128;
}
extern "C" int ktb200_softmax_attn_tiles(int heads, int kv_heads, int maps, int n_tokens, int n_seqs) {
    return n_seqs + n_tokens / (kMmaRows / maps / mma_heads_per_tile(heads / kv_heads));
}
extern "C" int ktb200_window_softmax_attn_uses_tensor_cores(int heads, int kv_heads, int dim, int vdim, int dtype) {
    return ktb200_softmax_attn_uses_tensor_cores(heads, kv_heads, 1, dim, vdim, dtype);
}
extern "C" int ktb200_window_softmax_attn_tiles(int heads, int kv_heads, int n_tokens, int n_seqs) { return ktb200_softmax_attn_tiles(heads, kv_heads, 1, n_tokens, n_seqs); }

extern "C" int ktb200_softmax_attn(const ktb200_softmax_attn_params* c, int n_tokens, int splits, float* workspace, int dtype, int allow_tensor_cores, void* stream) {
    if (!c || !c->q || !c->pos || !c->slot || !c->page_table || !c->cache || !c->out || c->heads <= 0 || c->kv_heads <= 0 || c->heads % c->kv_heads || c->maps < 1 || c->maps > 2 ||
        c->dim <= 0 || c->vdim <= 0 || c->vdim > 32 * kSmMaxCols || (c->maps == 2 && !c->lambda) || (c->dist_r1 && !c->dist_r2) || splits < 1 || c->page_size <= 0 || c->max_pages <= 0 ||
        c->out_stride < (long)c->heads * c->vdim) {
        set_error("softmax_attn: bad argument (value size <= %d)", 32 * kSmMaxCols);
        return KTB200_EINVAL;
    }
    if (n_tokens <= 0) return KTB200_OK;
    if (splits > kMergeMaxSplits) { set_error("softmax_attn: at most %d splits", kMergeMaxSplits); return KTB200_EINVAL; }
    const int heads = c->heads, kv_heads = c->kv_heads, dim = c->dim, vdim = c->vdim, maps = c->maps;
    const long rows = (long)n_tokens * heads;
    auto even = [](const void* p, long stride) { return (reinterpret_cast<uintptr_t>(p) & 3) == 0 && (stride & 1) == 0; };
    const bool tc = allow_tensor_cores && c->seqs && c->n_seqs > 0 && ktb200_softmax_attn_uses_tensor_cores(heads, kv_heads, maps, dim, vdim, dtype) &&
                    even(c->out, c->out_stride) && (!c->gate || even(c->gate, c->gate_stride));
    if (ktb200_softmax_attn_workspace(n_tokens, heads, maps, vdim, splits, tc) && !workspace) { set_error("softmax_attn: workspace missing"); return KTB200_EINVAL; }
    const bool merge = splits > 1 || (maps > 1 && !tc);
    SmAttn a{c->q, heads, kv_heads, maps, dim, vdim, c->scale, c->head_scale, c->softcap, c->window, c->chunk, c->dist_r1, c->dist_r2, c->sink, c->gate, c->gate_stride, c->out_scale,
             c->lambda, c->rms_eps, c->pos, c->slot, c->seqs, c->seqs_stride, c->n_seqs, 0, c->page_table, c->max_pages, c->page_size, c->cache, c->out, c->out_stride,
             merge ? workspace : nullptr, splits};
    if (tc) {
        using B = __nv_bfloat16;
        const int RH = a.RH = mma_heads_per_tile(heads / kv_heads), row_tile = kMmaRows / maps;
        const dim3 grid(ktb200_softmax_attn_tiles(heads, kv_heads, maps, n_tokens, c->n_seqs), kv_heads * (heads / kv_heads / RH), splits);
        const size_t smem = (((size_t)row_tile + 2 * kMmaKeys) * (maps * dim + kMmaPad) + (size_t)2 * kMmaKeys * (vdim + kMmaPad)) * sizeof(B);
#define MMA_LAUNCH(DK, DV, MAPS, BIAS)                                                                                             \
    do {                                                                                                                           \
        GRANT_SMEM((window_softmax_attn_mma_kernel<DK, DV, MAPS, BIAS>), smem);                                                    \
        window_softmax_attn_mma_kernel<DK, DV, MAPS, BIAS><<<grid, kMmaRows * 2, smem, (cudaStream_t)stream>>>(a);                 \
    } while (0)
#define MMA_SIZES(MAPS, BIAS)                                              \
    do {                                                                   \
        if (dim <= 64 && vdim <= 64) MMA_LAUNCH(4, 4, MAPS, BIAS);         \
        else if (dim <= 64) MMA_LAUNCH(4, 8, MAPS, BIAS);                  \
        else MMA_LAUNCH(8, 8, MAPS, BIAS);                                 \
    } while (0)
        if (maps == 1) {
            if (c->dist_r1) MMA_SIZES(1, true);
            else MMA_SIZES(1, false);
        } else {
            if (c->dist_r1) MMA_SIZES(2, true);
            else MMA_SIZES(2, false);
        }
#undef MMA_SIZES
#undef MMA_LAUNCH
        KTB_LAUNCH_CHECK();
        if (merge) {
            if (maps == 2) softmax_merge_kernel<B, 2><<<(unsigned)rows, 256, 0, (cudaStream_t)stream>>>(a);
            else softmax_merge_kernel<B, 1><<<(unsigned)rows, 128, 0, (cudaStream_t)stream>>>(a);
            KTB_LAUNCH_CHECK();
        }
        return KTB200_OK;
    }
    const int R = heads / kv_heads, HB = R < 8 ? R : 8, hblocks = (R + HB - 1) / HB;
    const size_t smem = ((size_t)HB * dim + (size_t)kSmTile * (dim + 1) + (size_t)kSmTile * vdim + (size_t)HB * kSmTile) * sizeof(float);
    if (smem > 200 * 1024) { set_error("softmax_attn: head too wide for shared memory"); return KTB200_EINVAL; }
    SEQ_DISPATCH(dtype, {
        GRANT_SMEM(window_softmax_attn_kernel<T>, smem);
        window_softmax_attn_kernel<T><<<dim3(n_tokens, kv_heads * maps * hblocks, splits), HB * 32, smem, (cudaStream_t)stream>>>(a);
        KTB_LAUNCH_CHECK();
        if (merge) {
            if (maps == 2) softmax_merge_kernel<T, 2><<<(unsigned)rows, 256, 0, (cudaStream_t)stream>>>(a);
            else softmax_merge_kernel<T, 1><<<(unsigned)rows, 128, 0, (cudaStream_t)stream>>>(a);
            KTB_LAUNCH_CHECK();
        }
    });
    return KTB200_OK;
}

extern "C" int ktb200_window_softmax_attn(const void* q, int heads, int kv_heads, int dim, int vdim, float scale, const float* head_scale, float softcap, int window, int chunk,
                                          const int* pos, const int* slot,
                                          const int* seqs, int seqs_stride, int n_seqs, const int* page_table, int max_pages, int page_size, const void* cache, void* out,
                                          int n_tokens, int splits, float* workspace, int dtype, int allow_tensor_cores, void* stream) {
    ktb200_softmax_attn_params c{};
    c.q = q; c.heads = heads; c.kv_heads = kv_heads; c.maps = 1; c.dim = dim; c.vdim = vdim; c.scale = scale; c.head_scale = head_scale; c.softcap = softcap; c.window = window; c.chunk = chunk;
    c.out_scale = 1.0f; c.pos = pos; c.slot = slot; c.seqs = seqs; c.seqs_stride = seqs_stride; c.n_seqs = n_seqs; c.page_table = page_table; c.max_pages = max_pages;
    c.page_size = page_size; c.cache = cache; c.out = out; c.out_stride = (long)heads * vdim;
    return ktb200_softmax_attn(&c, n_tokens, splits, workspace, dtype, allow_tensor_cores, stream);
}
