// Scans of mixers that carry a matrix S [D, Dv] per request and head from token to token, a column of S spread over many lanes:
// the form for portions of many tokens (single tokens and short portions, and delta-rule heads of few key channels: recurrent.cu).
//
//   WIDE_GATED_DELTA   S~ = diag(a) S, S' = S~ + k (b (v - S~^T k))^T, o = scale S'^T q   (a: a decay per key channel, b: a number)
//   WIDE_HEAD_DECAY    S' = c S + d k v^T, o = scale S'^T q                               (c, d: numbers per head)
//
// over the tokens of every segment, from and into the request's state slot, everything in float32.  The walk over the tokens is
// sequential; what makes it fast is that a token costs a lane little and waits for little:
//
// * KS lanes share NC neighbouring columns and hold R = 4 NI of their key channels each, as pairs; what a lane reads of a staged row serves all its columns, since reading the rows is what the walk is bound by.
//   Lane `part` holds the 16-byte groups part, part + KS, ... of a row, so that a staged row is a plain copy and its reads meet
//   no conflicts.
// * The delta rule reads the state along the key before it can write.  Written out, that read is a sum over the lanes that depends
//   on the write before it, and the chain sum - exchange - write would bound the walk.  The read of token t is therefore split:
//   S~_t^T k_t = (a_t k_t)^T S~_{t-1} + ((a_t k_t) . k_{t-1}) u_{t-1}, with u the values written.  The first part does not know
//   u_{t-1}, and its exchange runs while u_{t-1} is still being made; the number in front of u_{t-1} is the same for all columns
//   and is computed once per tile of tokens.
// * Read-outs of a group of tokens are summed over the lanes together: each exchange halves how many of them a lane still carries.
//
// Tiles of 32 tokens (the rows of q, k and decays, the block's values, the numbers per token) are staged in shared memory by
// asynchronous copies, the next one while this one is walked.  A tile's tokens are walked in groups; tokens beyond the
// segment's end are staged as ones that change nothing (a = 1, k = 0, b = 0).  A token's result does not depend on what else the
// step holds; where a request is cut, the split read of the cut's first token is one sum instead of two (float32 rounding).
// State layout: [slot, head, key channel, value channel].
#include "common.cuh"

enum { WIDE_GATED_DELTA = 0, WIDE_HEAD_DECAY = 1 };
constexpr int TILE = 32;
constexpr int DELTA_NC = 1, SPACE_NC = 2;                      // columns of a lane, as measured
__host__ __device__ constexpr int group_tokens(int nc) { return 16 / nc; }      // read-outs summed together: 16 of a lane's

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return make_float2(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y)); }
__device__ __forceinline__ float2 mul2(float2 a, float2 b) { return make_float2(a.x * b.x, a.y * b.y); }
__device__ __forceinline__ float sum_halves(float2 v) { return v.x + v.y; }

__device__ __forceinline__ void copy_async4(float* smem, const float* gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
}
__device__ __forceinline__ void copy_async16(float* smem, const float* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
__device__ __forceinline__ void copy_async_wait_all() { asm volatile("cp.async.wait_group 0;\n" ::: "memory"); }

// Where a step's rows lie: columns of float32 rows `rows` [T, C] and `gates` [T, gate_stride].
struct WideRows {
    const float* rows;
    const float* gates;
    int C, gate_stride;
    int q_col, k_col, v_col;       // first columns of the queries, keys (number h / qk_div of D each) and values (h of Dv)
    int row_col;                   // gated delta: first column in `gates` of the decays, H of D
    int s0_col, s1_col;            // in `gates`: gated delta b; head decay c and d - a number per head
    int qk_div;
    int wide_copies;               // every row of D starts on 16 bytes and D is a multiple of 4
};

// A buffer of TILE tokens: rows of q, k (and decays) of DP floats, then VC values a token, then two numbers a token.
__host__ __device__ constexpr int wide_parts(int mode) { return mode == WIDE_GATED_DELTA ? 3 : 2; }
__host__ __device__ constexpr int wide_buffer_floats(int mode, int DP, int VC) { return TILE * (wide_parts(mode) * DP + VC + 2); }

template <int NC> struct Columns { float v[NC]; };
template <int NC> __device__ __forceinline__ Columns<NC> load_columns(const float* p, int valid, bool aligned) {
    Columns<NC> c;
    if (aligned && valid >= NC) {
        if constexpr (NC == 4) {
            const float4 x = *reinterpret_cast<const float4*>(p);
            c.v[0] = x.x; c.v[1] = x.y; c.v[2] = x.z; c.v[3] = x.w;
        } else if constexpr (NC == 2) {
            const float2 x = *reinterpret_cast<const float2*>(p);
            c.v[0] = x.x; c.v[1] = x.y;
        } else {
            c.v[0] = *p;
        }
    } else {
#pragma unroll
        for (int i = 0; i < NC; ++i) c.v[i] = i < valid ? p[i] : 0.f;
    }
    return c;
}
template <int NC> __device__ __forceinline__ void store_columns(float* p, const Columns<NC>& c, int valid, bool aligned) {
    if (aligned && valid >= NC) {
        if constexpr (NC == 4) *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[1], c.v[2], c.v[3]);
        else if constexpr (NC == 2) *reinterpret_cast<float2*>(p) = make_float2(c.v[0], c.v[1]);
        else *p = c.v[0];
    } else {
#pragma unroll
        for (int i = 0; i < NC; ++i)
            if (i < valid) p[i] = c.v[i];
    }
}

// v[i] (i < N): this lane's shares of N sums over KS neighbouring lanes.  Afterwards the first max(1, N / KS) entries are
// whole sums; entry i is number `first` + i.
template <int N, int KS>
__device__ __forceinline__ int reduce_shares(float (&v)[N], int part) {
    int first = 0, left = N;
#pragma unroll
    for (int offset = (KS > N ? N : KS) / 2; offset >= 1; offset >>= 1) {
        const bool upper = part & offset;
        left >>= 1;
#pragma unroll
        for (int i = 0; i < N / 2; ++i)
            if (i < left) {
                const float mine = upper ? v[i + left] : v[i], other = upper ? v[i] : v[i + left];
                v[i] = mine + __shfl_xor_sync(0xffffffffu, other, offset);
            }
        if (upper) first += left;
    }
#pragma unroll
    for (int offset = N; offset < KS; offset <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], offset);
    return first;
}

// grid (column blocks, heads, segments); a warp holds 32 / KS groups of NC columns.
template <int MODE, int NI, int KS, int NC>
__global__ void __launch_bounds__(256) wide_scan_kernel(WideRows in, float q_scale, const int* __restrict__ seg_q_start,
                                                        const int* __restrict__ seg_q_len, const int* __restrict__ seg_slot,
                                                        float* __restrict__ memory, float* __restrict__ out, int H, int D, int Dv) {
    constexpr int NP = 2 * NI;                                 // pairs of key channels a lane holds of each of its columns
    constexpr int DP = 4 * NI * KS;                            // a staged row, zero beyond D
    constexpr int COLS = 32 / KS * NC;                         // columns of a warp
    constexpr int PARTS = wide_parts(MODE);
    constexpr int GROUP = group_tokens(NC);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int h = blockIdx.y, seg = blockIdx.z;
    const int part = lane % KS, VC = warps * COLS;
    const int my_col = warp * COLS + lane / KS * NC, col = blockIdx.x * VC + my_col;
    const int valid = Dv - col;                                // how many of the lane's columns exist, if fewer than NC
    const bool aligned = Dv % NC == 0;
    const int r0 = seg_q_start[seg], n = seg_q_len[seg], slot = seg_slot[seg];
    if (n <= 0) return;
    // The state was written by an earlier step (or zeroed at admission): it is on its way before the wait for this step's rows.
    float* mem = memory + ((size_t)slot * H + h) * D * Dv + col;
    auto channel = [&](int i) { return 4 * ((i >> 1) * KS + part) + 2 * (i & 1); };      // the first channel of pair i
    float2 S[NC][NP];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int d = channel(i);
        const Columns<NC> lo = load_columns<NC>(mem + (size_t)d * Dv, d < D ? valid : 0, aligned);
        const Columns<NC> hi = load_columns<NC>(mem + (size_t)(d + 1) * Dv, d + 1 < D ? valid : 0, aligned);
#pragma unroll
        for (int c = 0; c < NC; ++c) S[c][i] = make_float2(lo.v[c], hi.v[c]);
    }
    extern __shared__ __align__(16) float wide_s[];
    __shared__ float ahead_s[TILE];                            // gated delta: (a_t k_t) . k_{t-1}
    const int buffer_floats = wide_buffer_floats(MODE, DP, VC);
    if (D < DP)                                                // the channels beyond D
        for (int idx = threadIdx.x; idx < 2 * TILE * PARTS * (DP - D); idx += blockDim.x) {
            const int row = idx / (DP - D), d = D + idx - row * (DP - D);
            const int which = row >= TILE * PARTS;
            wide_s[(size_t)which * buffer_floats + (row - which * TILE * PARTS) * DP + d] = 0.f;
        }
    pdl_wait();
    pdl_launch_dependents();
    const int qk_off = h / in.qk_div * D;
    auto stage = [&](int which, int first_row, int count) {
        float* b = wide_s + (size_t)which * buffer_floats;
        float* v_b = b + TILE * PARTS * DP;
        float* s_b = v_b + TILE * VC;
        if (in.wide_copies) {
            const int per_row = D >> 2;
            for (int idx = threadIdx.x; idx < count * per_row; idx += blockDim.x) {
                const int row = idx / per_row, d = 4 * (idx - row * per_row);
                const float* src = in.rows + (size_t)(first_row + row) * in.C + qk_off + d;
                float* dst = b + row * DP + d;
                copy_async16(dst, src + in.q_col);
                copy_async16(dst + TILE * DP, src + in.k_col);
                if (MODE == WIDE_GATED_DELTA)
                    copy_async16(dst + 2 * TILE * DP, in.gates + (size_t)(first_row + row) * in.gate_stride + in.row_col + h * D + d);
            }
        } else {
            for (int idx = threadIdx.x; idx < count * D; idx += blockDim.x) {
                const int row = idx / D, d = idx - row * D;
                const float* src = in.rows + (size_t)(first_row + row) * in.C + qk_off + d;
                float* dst = b + row * DP + d;
                copy_async4(dst, src + in.q_col);
                copy_async4(dst + TILE * DP, src + in.k_col);
                if (MODE == WIDE_GATED_DELTA)
                    copy_async4(dst + 2 * TILE * DP, in.gates + (size_t)(first_row + row) * in.gate_stride + in.row_col + h * D + d);
            }
        }
        const int v_cols = min(VC, Dv - (int)blockIdx.x * VC);
        for (int idx = threadIdx.x; idx < count * v_cols; idx += blockDim.x) {
            const int row = idx / v_cols, c = idx - row * v_cols;
            copy_async4(v_b + row * VC + c, in.rows + (size_t)(first_row + row) * in.C + in.v_col + h * Dv + blockIdx.x * VC + c);
        }
        for (int row = threadIdx.x; row < count; row += blockDim.x) {
            const float* grow = in.gates + (size_t)(first_row + row) * in.gate_stride + h;
            copy_async4(s_b + row, grow + in.s0_col);
            if (MODE == WIDE_HEAD_DECAY) copy_async4(s_b + TILE + row, grow + in.s1_col);
        }
        copy_async_commit();
        // Tokens that change nothing, up to a whole group.
        const int padded = (count + GROUP - 1) / GROUP * GROUP;
        for (int idx = threadIdx.x; idx < (padded - count) * DP; idx += blockDim.x) {
            float* dst = b + count * DP + idx;
            dst[0] = 0.f;
            dst[TILE * DP] = 0.f;
            if (MODE == WIDE_GATED_DELTA) dst[2 * TILE * DP] = 1.f;
        }
        for (int idx = threadIdx.x; idx < (padded - count) * VC; idx += blockDim.x) v_b[count * VC + idx] = 0.f;
        for (int row = count + threadIdx.x; row < padded; row += blockDim.x) {
            s_b[row] = MODE == WIDE_GATED_DELTA ? 0.f : 1.f;
            s_b[TILE + row] = 0.f;
        }
    };
    stage(0, r0, min(TILE, n));
    float shares[GROUP * NC];                                  // read-outs of a group's tokens: this lane's shares
    auto flush = [&](int first_token, int count) {             // `count` of the group's tokens exist
        float v[GROUP * NC];
#pragma unroll
        for (int i = 0; i < GROUP * NC; ++i) v[i] = shares[i];
        const int at = reduce_shares<GROUP * NC, KS>(v, part);
        constexpr int WHOLE = GROUP * NC > KS ? GROUP * NC / KS : 1;
        if (part < GROUP * NC) {
#pragma unroll
            for (int i = 0; i < WHOLE; ++i) {
                const int token = (at + i) / NC, c = (at + i) % NC;
                if (token < count && c < valid) out[((size_t)(r0 + first_token + token) * H + h) * Dv + col + c] = v[i] * q_scale;
            }
        }
    };
    // Gated delta: S holds S~ of the token before (its write still to be added), `wrote` what it writes, k_before its key.
    float2 k_before[NP], q_before[NP];
    float wrote[NC];
#pragma unroll
    for (int i = 0; i < NP; ++i) k_before[i] = q_before[i] = make_float2(0.f, 0.f);
#pragma unroll
    for (int c = 0; c < NC; ++c) wrote[c] = 0.f;
    for (int t0 = 0; t0 < n; t0 += TILE) {
        const int which = (t0 / TILE) & 1, count = min(TILE, n - t0);
        const float* b = wide_s + (size_t)which * buffer_floats;
        const float* v_b = b + TILE * PARTS * DP + my_col;
        const float* s_b = b + TILE * PARTS * DP + TILE * VC;
        copy_async_wait_all();
        __syncthreads();                                       // this tile has landed; the one before has been walked
        if (MODE == WIDE_GATED_DELTA) {
            const float* last = wide_s + (size_t)(which ^ 1) * buffer_floats + TILE * DP + (TILE - 1) * DP;
            for (int tt = warp; tt < (count + GROUP - 1) / GROUP * GROUP; tt += warps) {
                const float* k = b + TILE * DP + tt * DP;
                const float* a = k + TILE * DP;
                const float* before = tt > 0 ? k - DP : last;
                float c = 0.f;
                if (tt > 0 || t0 > 0)
                    for (int d = lane; d < DP; d += 32) c = fmaf(a[d] * k[d], before[d], c);
                c = warp_sum(c);
                if (lane == 0) ahead_s[tt] = c;
            }
            __syncthreads();
        }
        if (t0 + TILE < n) stage(which ^ 1, r0 + t0 + TILE, min(TILE, n - t0 - TILE));
#pragma unroll 1
        for (int g = 0; g < count; g += GROUP) {
#pragma unroll
            for (int j = 0; j < GROUP; ++j) {
                const int tt = g + j;
                const float4* q4 = reinterpret_cast<const float4*>(b + tt * DP) + part;
                const float4* k4 = q4 + TILE * DP / 4;
                float2 q[NP], k[NP];
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const float4 kk = k4[i * KS], qq = q4[i * KS];
                    k[2 * i] = make_float2(kk.x, kk.y); k[2 * i + 1] = make_float2(kk.z, kk.w);
                    q[2 * i] = make_float2(qq.x, qq.y); q[2 * i + 1] = make_float2(qq.z, qq.w);
                }
                const Columns<NC> v = load_columns<NC>(v_b + tt * VC, NC, true);
                if (MODE == WIDE_GATED_DELTA) {
                    const float4* a4 = k4 + TILE * DP / 4;
                    float2 a[NP], w[NP];
#pragma unroll
                    for (int i = 0; i < NI; ++i) {
                        const float4 aa = a4[i * KS];
                        a[2 * i] = make_float2(aa.x, aa.y); a[2 * i + 1] = make_float2(aa.z, aa.w);
                        w[2 * i] = mul2(a[2 * i], k[2 * i]);
                        w[2 * i + 1] = mul2(a[2 * i + 1], k[2 * i + 1]);
                    }
                    float read[NC];
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        float2 p0 = mul2(w[0], S[c][0]), p1 = mul2(w[1], S[c][1]);
#pragma unroll
                        for (int i = 2; i < NP; i += 2) {
                            p0 = fma2(w[i], S[c][i], p0);
                            p1 = fma2(w[i + 1], S[c][i + 1], p1);
                        }
                        read[c] = sum_halves(p0) + sum_halves(p1);
                    }
#pragma unroll
                    for (int offset = KS / 2; offset >= 1; offset >>= 1)
#pragma unroll
                        for (int c = 0; c < NC; ++c) read[c] += __shfl_xor_sync(0xffffffffu, read[c], offset);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        const float2 w2 = make_float2(wrote[c], wrote[c]);
                        float2 o0 = make_float2(0.f, 0.f), o1 = make_float2(0.f, 0.f);
#pragma unroll
                        for (int i = 0; i < NP; i += 2) {
                            S[c][i] = fma2(k_before[i], w2, S[c][i]);    // the token before, whole
                            S[c][i + 1] = fma2(k_before[i + 1], w2, S[c][i + 1]);
                            o0 = fma2(q_before[i], S[c][i], o0);
                            o1 = fma2(q_before[i + 1], S[c][i + 1], o1);
                            S[c][i] = mul2(a[i], S[c][i]);
                            S[c][i + 1] = mul2(a[i + 1], S[c][i + 1]);
                        }
                        shares[(j + GROUP - 1) % GROUP * NC + c] = sum_halves(o0) + sum_halves(o1);
                    }
                    if (j == 0 && t0 + g > 0) flush(t0 + g - GROUP, GROUP);
#pragma unroll
                    for (int c = 0; c < NC; ++c) wrote[c] = s_b[tt] * (v.v[c] - fmaf(ahead_s[tt], wrote[c], read[c]));
#pragma unroll
                    for (int i = 0; i < NP; ++i) {
                        k_before[i] = k[i];
                        q_before[i] = q[i];
                    }
                } else {
                    const float keep = s_b[tt], take = s_b[TILE + tt];
                    const float2 keep2 = make_float2(keep, keep);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        const float gain = take * v.v[c];
                        const float2 gain2 = make_float2(gain, gain);
                        float2 o0 = make_float2(0.f, 0.f), o1 = make_float2(0.f, 0.f);
#pragma unroll
                        for (int i = 0; i < NP; i += 2) {
                            S[c][i] = fma2(keep2, S[c][i], mul2(k[i], gain2));
                            S[c][i + 1] = fma2(keep2, S[c][i + 1], mul2(k[i + 1], gain2));
                            o0 = fma2(q[i], S[c][i], o0);
                            o1 = fma2(q[i + 1], S[c][i + 1], o1);
                        }
                        shares[j * NC + c] = sum_halves(o0) + sum_halves(o1);
                    }
                }
            }
            if (MODE == WIDE_HEAD_DECAY) flush(t0 + g, count - g);
        }
    }
    if (MODE == WIDE_GATED_DELTA) {                            // the last token's write and read-out
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const float2 w2 = make_float2(wrote[c], wrote[c]);
            float2 o0 = make_float2(0.f, 0.f), o1 = make_float2(0.f, 0.f);
#pragma unroll
            for (int i = 0; i < NP; i += 2) {
                S[c][i] = fma2(k_before[i], w2, S[c][i]);
                S[c][i + 1] = fma2(k_before[i + 1], w2, S[c][i + 1]);
                o0 = fma2(q_before[i], S[c][i], o0);
                o1 = fma2(q_before[i + 1], S[c][i + 1], o1);
            }
            shares[(GROUP - 1) * NC + c] = sum_halves(o0) + sum_halves(o1);
        }
        const int first = (n - 1) / GROUP * GROUP;
        flush(first, n - first);
    }
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int d = channel(i);
        Columns<NC> lo, hi;
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            lo.v[c] = S[c][i].x;
            hi.v[c] = S[c][i].y;
        }
        store_columns<NC>(mem + (size_t)d * Dv, lo, d < D ? valid : 0, aligned);
        store_columns<NC>(mem + (size_t)(d + 1) * Dv, hi, d + 1 < D ? valid : 0, aligned);
    }
}

template <int MODE, int NI, int KS, int NC>
static int launch_wide(const WideRows& in, float q_scale, const int* seg_q_start, const int* seg_q_len, const int* seg_slot, float* memory,
                       float* out, int S, int H, int D, int Dv, cudaStream_t stream) {
    constexpr int COLS = 32 / KS * NC, DP = 4 * NI * KS;
    const int total = (Dv + COLS - 1) / COLS;                  // warps a head takes
    // Many warps share a staged row, but every SM wants a block: fewer warps a block where that brings more blocks.
    int warps = 8;
    auto blocks = [&](int w) { return (long long)S * H * ((total + w - 1) / w); };
    while (warps > 1 && (warps / 2 >= total || blocks(warps) < kvb_sm_count() * 3 / 4)) warps >>= 1;
    auto bytes = [&](int w) { return 2 * (size_t)wide_buffer_floats(MODE, DP, w * COLS) * sizeof(float); };
    if (bytes(warps) > 220 * 1024) return KVB_ERR_LIMIT;
    if (bytes(warps) > 46 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(wide_scan_kernel<MODE, NI, KS, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes(warps));
        if (e != cudaSuccess) return (int)e;
    }
    kvb_launch(wide_scan_kernel<MODE, NI, KS, NC>, dim3((total + warps - 1) / warps, H, S), dim3(32 * warps), bytes(warps), stream, in, q_scale,
               seg_q_start, seg_q_len, seg_slot, memory, out, H, D, Dv);
    return kvb_launch_status();
}

// rows: float32 [T, C] = [q: G heads of D | k: G heads of D | v: H heads of Dv], unit vectors and values as the delta rule wants them;
// gates: float32 [T, gate_stride] = [decays: H of D | b: H | ...].  Head h reads query and key h / (H / G).
KVB_API int kvb_gated_delta_scan_wide(const float* rows, const float* gates, int gate_stride, float q_scale, const int* seg_q_start,
                                 const int* seg_q_len, const int* seg_slot, float* memory, float* out, int S, int H, int G, int D, int Dv,
                                 cudaStream_t stream) {
    if (S <= 0) return KVB_OK;
    if (H < 1 || G < 1 || H % G || D < 1 || Dv < 1 || gate_stride < H * D + H) return KVB_ERR_SHAPE;
    if (D > 256 || H > 65535 || S > 65535) return KVB_ERR_LIMIT;
    const int C = 2 * G * D + H * Dv;
    const bool wide = ((D | C | gate_stride) & 3) == 0 && (((uintptr_t)rows | (uintptr_t)gates) & 15) == 0;
    const WideRows in = {rows, gates, C, gate_stride, 0, G * D, 2 * G * D, 0, H * D, 0, H / G, wide ? 1 : 0};
#define KVB_WIDE(NI, KS) launch_wide<WIDE_GATED_DELTA, NI, KS, DELTA_NC>(in, q_scale, seg_q_start, seg_q_len, seg_slot, memory, out, S, H, D, Dv, stream)
    if (D <= 32) return KVB_WIDE(2, 4);
    if (D <= 64) return KVB_WIDE(2, 8);
    if (D <= 128) return KVB_WIDE(2, 16);
    return KVB_WIDE(2, 32);
#undef KVB_WIDE
}

// rows: float32 [T, C] = [x: H heads of Dv | B: G of N | C: G of N]; gates: float32 [T, 2 H] = [decay: H | d: H].  Head h reads B and C
// of group h / (H / G): S' = decay S + d B x^T, out = S'^T C.
KVB_API int kvb_state_space_scan_wide(const float* rows, const float* gates, const int* seg_q_start, const int* seg_q_len, const int* seg_slot,
                                 float* memory, float* out, int S, int H, int G, int N, int Dv, cudaStream_t stream) {
    if (S <= 0) return KVB_OK;
    if (H < 1 || G < 1 || H % G || N < 1 || Dv < 1) return KVB_ERR_SHAPE;
    if (N > 256 || H > 65535 || S > 65535) return KVB_ERR_LIMIT;
    const int C = H * Dv + 2 * G * N;
    const bool wide = ((N | C | (H * Dv)) & 3) == 0 && ((uintptr_t)rows & 15) == 0;
    const WideRows in = {rows, gates, C, 2 * H, H * Dv + G * N, H * Dv, 0, 0, 0, H, H / G, wide ? 1 : 0};
#define KVB_WIDE(NI, KS) launch_wide<WIDE_HEAD_DECAY, NI, KS, SPACE_NC>(in, 1.f, seg_q_start, seg_q_len, seg_slot, memory, out, S, H, N, Dv, stream)
    if (N <= 32) return KVB_WIDE(2, 4);
    if (N <= 64) return KVB_WIDE(2, 8);
    if (N <= 128) return KVB_WIDE(2, 16);
    return KVB_WIDE(2, 32);
#undef KVB_WIDE
}
