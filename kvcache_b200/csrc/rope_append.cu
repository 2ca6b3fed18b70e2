// Bias + rotation of queries and keys + append of keys and values into cache pages, one kernel.
//
// Replaces k_add_bias, k_rope / k_rope_pos and k_write_kv / k_batched_write_kv of the
// reference (src/qwen_kernels.cu:46-52, :65-81, :253-267, :111-126, :270-290): the
// projection's output is read once, the bias is added and the pair (t, t + rot/2) is
// rotated in float32, and the result is rounded once on its way to the query buffer or
// to the page `block_table[segment][pos / page]`, slot `pos % page`
// (pool layout [pages, kv_heads, page, head_dim] as src/include/kv_cache_manager.h:89-91).
//
// The angles come from a table cos/sin[pos, t] that the host fills in double
// precision; a position beyond the table sets the error word.
#include "common.cuh"

template <typename T>
__global__ void qkv_rope_append_kernel(const T* __restrict__ qkv, const float* __restrict__ bias,
                                       const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                       int rot_half, int table_len, const int* __restrict__ positions,
                                       const int* __restrict__ row_segment, const int* __restrict__ block_table,
                                       int table_stride, T* __restrict__ k_pages, T* __restrict__ v_pages,
                                       T* __restrict__ q_out, int Hq, int Hkv, int D, int page_size, int write_kv,
                                       int* __restrict__ err) {
    pdl_wait();
    pdl_launch_dependents();
    const int r = blockIdx.x;
    const int width = (Hq + 2 * Hkv) * D;
    const int pos = positions[r];
    const T* src = qkv + (size_t)r * width;
    const int rot = 2 * rot_half;

    size_t page_base = 0;
    bool page_ok = true;
    if (write_kv) {
        const int seg = row_segment[r];
        const int page = block_table[(size_t)seg * table_stride + pos / page_size];
        if (page < 0) {
            page_ok = false;
            if (threadIdx.x == 0) atomicOr(err, KVB_DEV_BAD_PAGE);
        }
        page_base = (size_t)(page < 0 ? 0 : page) * Hkv * page_size * D + (size_t)(pos % page_size) * D;
    }
    const bool pos_ok = rot_half == 0 || (pos >= 0 && pos < table_len);
    if (!pos_ok && threadIdx.x == 0) atomicOr(err, KVB_DEV_BAD_POS);
    const float* cr = cos_t + (size_t)(pos_ok ? pos : 0) * rot_half;
    const float* sr = sin_t + (size_t)(pos_ok ? pos : 0) * rot_half;

    for (int idx = threadIdx.x; idx < width; idx += blockDim.x) {
        const int head = idx / D, d = idx - head * D;
        float x = to_f32<T>(src[idx]);
        if (bias) x += bias[idx];
        const bool is_v = head >= Hq + Hkv;
        if (!is_v && d < rot) {
            // rotate-half pairing (t, t + rot/2): x'_t = x_t cos - x_p sin ; x'_p = x_p cos + x_t sin
            const bool low = d < rot_half;
            const int t = low ? d : d - rot_half;
            const int pidx = low ? idx + rot_half : idx - rot_half;
            float xp = to_f32<T>(src[pidx]);
            if (bias) xp += bias[pidx];
            const float c = cr[t], s = sr[t];
            x = low ? (x * c - xp * s) : (x * c + xp * s);
        }
        if (head < Hq) {
            q_out[(size_t)r * Hq * D + idx] = from_f32<T>(x);
        } else if (write_kv && page_ok) {
            const int hk = is_v ? head - Hq - Hkv : head - Hq;
            const size_t dst = page_base + (size_t)hk * page_size * D + d;
            (is_v ? v_pages : k_pages)[dst] = from_f32<T>(x);
        }
    }
}

// bfloat16, head sizes and rotation halves that are multiples of 8: one thread moves 8 elements
// (16 bytes) of a head; for a rotated chunk it also reads the partner chunk rot/2 further (or back).
// What does not depend on the product before this kernel - the row's position and page, and the first
// chunk's angles and biases - is read before the wait for that product.
struct ChunkTables {
    float cs[8], sn[8], b_self[8], b_partner[8];
};

__device__ __forceinline__ void chunk_tables(ChunkTables& t, int c, int chunks_per_head, int D, int Hq, int Hkv, int rot_half,
                                             const float* cr, const float* sr, const float* bias) {
    const int head = c / chunks_per_head, d = (c - head * chunks_per_head) * 8;
    const int idx = head * D + d;
    const bool rotated = head < Hq + Hkv && d < 2 * rot_half;
    const bool low = d < rot_half;
    const int t0 = low ? d : d - rot_half;
    const int pidx = low ? idx + rot_half : idx - rot_half;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        t.b_self[k] = bias ? bias[idx + k] : 0.f;
        t.b_partner[k] = (bias && rotated) ? bias[pidx + k] : 0.f;
        t.cs[k] = rotated ? cr[t0 + k] : 1.f;
        t.sn[k] = rotated ? sr[t0 + k] : 0.f;
    }
}

__global__ void qkv_rope_append_vec8_kernel(const bf16* __restrict__ qkv, const float* __restrict__ bias,
                                            const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                            int rot_half, int table_len, const int* __restrict__ positions,
                                            const int* __restrict__ row_segment, const int* __restrict__ block_table,
                                            int table_stride, bf16* __restrict__ k_pages, bf16* __restrict__ v_pages,
                                            bf16* __restrict__ q_out, int Hq, int Hkv, int D, int page_size, int write_kv,
                                            int* __restrict__ err) {
    // This kernel is a few small blocks: it lets its successor (attention, which fetches block tables and old keys
    // before its own wait) onto the SMs at once, while the product before this kernel may still be running.
    pdl_launch_dependents();
    const int r = blockIdx.x;
    const int width = (Hq + 2 * Hkv) * D;
    const int pos = positions[r];
    const int rot = 2 * rot_half;
    size_t page_base = 0;
    bool page_ok = true;
    if (write_kv) {
        const int seg = row_segment[r];
        const int page = block_table[(size_t)seg * table_stride + pos / page_size];
        if (page < 0) {
            page_ok = false;
            if (threadIdx.x == 0) atomicOr(err, KVB_DEV_BAD_PAGE);
        }
        page_base = (size_t)(page < 0 ? 0 : page) * Hkv * page_size * D + (size_t)(pos % page_size) * D;
    }
    const bool pos_ok = rot_half == 0 || (pos >= 0 && pos < table_len);
    if (!pos_ok && threadIdx.x == 0) atomicOr(err, KVB_DEV_BAD_POS);
    const float* cr = cos_t + (size_t)(pos_ok ? pos : 0) * rot_half;
    const float* sr = sin_t + (size_t)(pos_ok ? pos : 0) * rot_half;
    const int chunks_per_head = D >> 3;
    const int chunks = width >> 3;
    ChunkTables tab;
    if ((int)threadIdx.x < chunks) chunk_tables(tab, threadIdx.x, chunks_per_head, D, Hq, Hkv, rot_half, cr, sr, bias);
    pdl_wait();
    const bf16* src = qkv + (size_t)r * width;
    for (int c = threadIdx.x; c < chunks; c += blockDim.x) {
        if (c != (int)threadIdx.x) chunk_tables(tab, c, chunks_per_head, D, Hq, Hkv, rot_half, cr, sr, bias);
        const int head = c / chunks_per_head, d = (c - head * chunks_per_head) * 8;
        const int idx = head * D + d;
        float x[8];
        {
            const uint4 raw = *reinterpret_cast<const uint4*>(src + idx);
            const uint32_t wv[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&wv[k]));
                x[2 * k] = f.x; x[2 * k + 1] = f.y;
            }
            if (bias) {
#pragma unroll
                for (int k = 0; k < 8; ++k) x[k] += tab.b_self[k];
            }
        }
        const bool is_v = head >= Hq + Hkv;
        if (!is_v && d < rot) {
            const bool low = d < rot_half;
            const int pidx = low ? idx + rot_half : idx - rot_half;
            const uint4 raw = *reinterpret_cast<const uint4*>(src + pidx);
            const uint32_t wv[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&wv[k]));
                float xp0 = f.x, xp1 = f.y;
                if (bias) { xp0 += tab.b_partner[2 * k]; xp1 += tab.b_partner[2 * k + 1]; }
                const float c0 = tab.cs[2 * k], s0 = tab.sn[2 * k], c1 = tab.cs[2 * k + 1], s1 = tab.sn[2 * k + 1];
                x[2 * k] = low ? (x[2 * k] * c0 - xp0 * s0) : (x[2 * k] * c0 + xp0 * s0);
                x[2 * k + 1] = low ? (x[2 * k + 1] * c1 - xp1 * s1) : (x[2 * k + 1] * c1 + xp1 * s1);
            }
        }
        uint32_t ow[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            __nv_bfloat162 o = __floats2bfloat162_rn(x[2 * k], x[2 * k + 1]);
            ow[k] = *reinterpret_cast<uint32_t*>(&o);
        }
        const uint4 packed = make_uint4(ow[0], ow[1], ow[2], ow[3]);
        if (head < Hq) {
            *reinterpret_cast<uint4*>(q_out + (size_t)r * Hq * D + idx) = packed;
        } else if (write_kv && page_ok) {
            const int hk = is_v ? head - Hq - Hkv : head - Hq;
            *reinterpret_cast<uint4*>((is_v ? v_pages : k_pages) + page_base + (size_t)hk * page_size * D + d) = packed;
        }
    }
}

// The same for steps of many rows (portions of prompts): a block takes ROWS consecutive rows.  Their positions and
// pages are looked up and their angles staged in shared memory once, before the wait (a row's 2 * rot_half angles are
// the same for all its heads); a thread keeps the biases of its chunk, which are the same for every row, in
// registers, and the loads of all ROWS rows of its chunk are in flight together.  With a quarter of the blocks of
// the one-row kernel the whole grid is on the SMs at once.
template <int ROWS>
__global__ void qkv_rope_append_rows_kernel(const bf16* __restrict__ qkv, const float* __restrict__ bias,
                                            const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                            int rot_half, int table_len, const int* __restrict__ positions,
                                            const int* __restrict__ row_segment, const int* __restrict__ block_table,
                                            int table_stride, bf16* __restrict__ k_pages, bf16* __restrict__ v_pages,
                                            bf16* __restrict__ q_out, int T, int Hq, int Hkv, int D, int page_size,
                                            int write_kv, int* __restrict__ err) {
    extern __shared__ float angles[];                      // [ROWS][2][rot_half]: cos, sin
    __shared__ long long page_base_s[ROWS];                // element offset of the row's slot in the pools; -1: no page
    const int r0 = blockIdx.x * ROWS;
    const int width = (Hq + 2 * Hkv) * D;
    const int rot = 2 * rot_half;
    if (threadIdx.x < ROWS) {
        const int r = r0 + threadIdx.x;
        long long base = -1;
        if (r < T && write_kv) {
            const int pos = positions[r];
            const int page = block_table[(size_t)row_segment[r] * table_stride + pos / page_size];
            if (page < 0) atomicOr(err, KVB_DEV_BAD_PAGE);
            else base = (long long)page * Hkv * page_size * D + (long long)(pos % page_size) * D;
        }
        page_base_s[threadIdx.x] = base;
    }
    for (int i = threadIdx.x; i < ROWS * rot; i += blockDim.x) {
        const int row = i / rot, j = i - row * rot, r = r0 + row;
        float v = j < rot_half ? 1.f : 0.f;
        if (r < T) {
            const int pos = positions[r];
            const bool pos_ok = pos >= 0 && pos < table_len;
            if (!pos_ok && j == 0) atomicOr(err, KVB_DEV_BAD_POS);
            const int p = pos_ok ? pos : 0;
            v = j < rot_half ? cos_t[(size_t)p * rot_half + j] : sin_t[(size_t)p * rot_half + j - rot_half];
        }
        angles[i] = v;
    }
    const int chunks_per_head = D >> 3;
    const int chunks = width >> 3;
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    for (int c = threadIdx.x; c < chunks; c += blockDim.x) {
        const int head = c / chunks_per_head, d = (c - head * chunks_per_head) * 8;
        const int idx = head * D + d;
        const bool is_v = head >= Hq + Hkv;
        const bool rotated = !is_v && d < rot;
        const bool low = d < rot_half;
        const int t0 = low ? d : d - rot_half;
        const int pidx = low ? idx + rot_half : idx - rot_half;
        float b_self[8], b_partner[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            b_self[k] = bias ? bias[idx + k] : 0.f;
            b_partner[k] = (bias && rotated) ? bias[pidx + k] : 0.f;
        }
        uint4 own[ROWS], partner[ROWS];
#pragma unroll
        for (int row = 0; row < ROWS; ++row) {
            const int r = min(r0 + row, T - 1);
            own[row] = *reinterpret_cast<const uint4*>(qkv + (size_t)r * width + idx);
            partner[row] = rotated ? *reinterpret_cast<const uint4*>(qkv + (size_t)r * width + pidx) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int row = 0; row < ROWS; ++row) {
            const int r = r0 + row;
            if (r >= T) break;
            const uint32_t wv[4] = {own[row].x, own[row].y, own[row].z, own[row].w};
            const uint32_t pv[4] = {partner[row].x, partner[row].y, partner[row].z, partner[row].w};
            const float* cs = angles + row * rot + t0;
            const float* sn = cs + rot_half;
            uint32_t ow[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&wv[k]));
                float x0 = f.x + b_self[2 * k], x1 = f.y + b_self[2 * k + 1];
                if (rotated) {
                    const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&pv[k]));
                    const float xp0 = g.x + b_partner[2 * k], xp1 = g.y + b_partner[2 * k + 1];
                    const float c0 = cs[2 * k], s0 = sn[2 * k], c1 = cs[2 * k + 1], s1 = sn[2 * k + 1];
                    x0 = low ? (x0 * c0 - xp0 * s0) : (x0 * c0 + xp0 * s0);
                    x1 = low ? (x1 * c1 - xp1 * s1) : (x1 * c1 + xp1 * s1);
                }
                __nv_bfloat162 o = __floats2bfloat162_rn(x0, x1);
                ow[k] = *reinterpret_cast<uint32_t*>(&o);
            }
            const uint4 packed = make_uint4(ow[0], ow[1], ow[2], ow[3]);
            if (head < Hq) {
                *reinterpret_cast<uint4*>(q_out + (size_t)r * Hq * D + idx) = packed;
            } else if (write_kv && page_base_s[row] >= 0) {
                const int hk = is_v ? head - Hq - Hkv : head - Hq;
                *reinterpret_cast<uint4*>((is_v ? v_pages : k_pages) + page_base_s[row] + (size_t)hk * page_size * D + d) = packed;
            }
        }
    }
}

KVB_API int kvb_qkv_rope_append(int dtype, const void* qkv, const float* bias, const float* cos_t,
                                const float* sin_t, int rot_half, int table_len, const int* positions,
                                const int* row_segment, const int* block_table, int table_stride, void* k_pages,
                                void* v_pages, void* q_out, int T, int Hq, int Hkv, int D, int page_size,
                                int write_kv, int* err, cudaStream_t stream) {
    if (T <= 0) return KVB_OK;
    if (2 * rot_half > D || rot_half < 0) return KVB_ERR_SHAPE;
    const int width = (Hq + 2 * Hkv) * D;
    const int threads = width >= 1024 ? 256 : 128;
    const uintptr_t addresses = (uintptr_t)qkv | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)q_out;
    if (dtype == KVB_BF16 && D % 8 == 0 && rot_half % 8 == 0 && (addresses & 15) == 0) {
        const int chunk_threads = width / 8 >= 1024 ? 1024 : (width / 8 + 31) / 32 * 32;
        if (T >= 256 && rot_half > 0) {
            constexpr int ROWS = 4;
            kvb_launch(qkv_rope_append_rows_kernel<ROWS>, dim3((T + ROWS - 1) / ROWS), dim3(chunk_threads),
                       (size_t)ROWS * 2 * rot_half * sizeof(float), stream, (const bf16*)qkv, bias, cos_t, sin_t, rot_half, table_len,
                       positions, row_segment, block_table, table_stride, (bf16*)k_pages, (bf16*)v_pages, (bf16*)q_out, T, Hq,
                       Hkv, D, page_size, write_kv, err);
            return kvb_launch_status();
        }
        // One 16-byte chunk per thread where the row allows it.
        kvb_launch(qkv_rope_append_vec8_kernel, dim3(T), dim3(width / 8 >= 1024 ? 1024 : (width / 8 + 31) / 32 * 32), 0, stream,
            (const bf16*)qkv, bias, cos_t, sin_t, rot_half, table_len, positions, row_segment, block_table, table_stride,
            (bf16*)k_pages, (bf16*)v_pages, (bf16*)q_out, Hq, Hkv, D, page_size, write_kv, err);
        return kvb_launch_status();
    }
    if (dtype == KVB_F32)
        kvb_launch(qkv_rope_append_kernel<float>, dim3(T), dim3(threads), 0, stream, 
            (const float*)qkv, bias, cos_t, sin_t, rot_half, table_len, positions, row_segment, block_table,
            table_stride, (float*)k_pages, (float*)v_pages, (float*)q_out, Hq, Hkv, D, page_size, write_kv, err);
    else if (dtype == KVB_BF16)
        kvb_launch(qkv_rope_append_kernel<bf16>, dim3(T), dim3(threads), 0, stream, 
            (const bf16*)qkv, bias, cos_t, sin_t, rot_half, table_len, positions, row_segment, block_table,
            table_stride, (bf16*)k_pages, (bf16*)v_pages, (bf16*)q_out, Hq, Hkv, D, page_size, write_kv, err);
    else
        return KVB_ERR_DTYPE;
    return kvb_launch_status();
}

// The same for layers whose queries and keys are normalised per head before the rotation, whose values have another
// size than their keys, or whose projection carries further columns: rows of `qkv` are
// [Hq heads of D | Hkv heads of D | Hkv heads of Dv | ...] with stride `row_stride`.  A query or key head becomes
// x / sqrt(mean(x^2) + eps) * w (w: D numbers shared by the heads; null: as it is), then its first 2 * rot_half numbers
// are rotated.  One block per row, a warp per head in turn; the normalised head passes through shared memory so that a
// lane finds its rotation partner.  Value pages are [pages, Hkv, page_size, Dv].  `Dk` >= D: queries and keys are stored
// Dk wide with zeros after their D numbers (keys as wide as values, so that kernels for equal sizes serve them; the
// zeros add nothing to a score).  `Dvs` >= Dv: values are stored Dvs wide with zeros after their Dv numbers.  `qt_every` > 0:
// the queries of a row at position p are multiplied by 1 + qt_coef * ln(floor((p + 1) / qt_every) + 1) (float32), after
// norm and rotation.  Hkv 0 (without write_kv): rows of queries alone, for a layer that reads another layer's keys.
enum { QKV_NORM = 1, QKV_NORM_ALL = 2, QKV_NORM_AFTER = 4 };
enum { QKV_MIX_NONE = 0, QKV_MIX_SOURCE = 1, QKV_MIX_BLEND = 2 };

template <typename T>
__global__ void qkv_norm_rope_append_kernel(const T* __restrict__ qkv, int row_stride, const float* __restrict__ bias,
                                            const float* __restrict__ q_w, const float* __restrict__ k_w, float eps, int norm_flags,
                                            const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_half,
                                            int table_len, const int* __restrict__ positions, const int* __restrict__ row_segment,
                                            const int* __restrict__ block_table, int table_stride, T* __restrict__ k_pages,
                                            T* __restrict__ v_pages, T* __restrict__ q_out, int Hq, int Hkv, int D, int Dv, int Dk,
                                            int page_size, int write_kv, int mix_mode, T* __restrict__ kept,
                                            const float* __restrict__ lam, int Dvs, float qt_coef, int qt_every,
                                            int* __restrict__ err) {
    extern __shared__ float head_s[];          // [warps][2][D], then 33 of scratch for the block sums
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    float* scratch = head_s + (size_t)warps * 2 * D;
    const bool normed = norm_flags & QKV_NORM, whole = norm_flags & QKV_NORM_ALL, after = norm_flags & QKV_NORM_AFTER;
    const int r = blockIdx.x;
    const int pos = positions[r];
    long long page_row = -1;                   // (page, slot) of the row's keys and values, counted in tokens
    if (write_kv) {
        const int page = block_table[(size_t)row_segment[r] * table_stride + pos / page_size];
        if (page < 0) {
            if (threadIdx.x == 0) atomicOr(err, KVB_DEV_BAD_PAGE);
        } else {
            page_row = (long long)page * Hkv * page_size + (pos % page_size);
        }
    }
    const bool pos_ok = rot_half == 0 || (pos >= 0 && pos < table_len);
    if (!pos_ok && threadIdx.x == 0) atomicOr(err, KVB_DEV_BAD_POS);
    const float* cr = cos_t + (size_t)(pos_ok ? pos : 0) * rot_half;
    const float* sr = sin_t + (size_t)(pos_ok ? pos : 0) * rot_half;
    const float mix = (mix_mode == QKV_MIX_BLEND) ? lam[0] : 0.f;
    const float q_gain = qt_every > 0 ? 1.f + qt_coef * logf((float)((pos + 1) / qt_every) + 1.f) : 1.f;
    pdl_wait();
    pdl_launch_dependents();
    const T* src = qkv + (size_t)r * row_stride;
    // A norm over the whole projection (before the rotation): one sum of squares for the row's queries, one for its keys.
    float inv_q = 1.f, inv_k = 1.f;
    if (normed && whole) {
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x; i < Hq * D; i += blockDim.x) {
            const float v = to_f32<T>(src[i]) + (bias ? bias[i] : 0.f);
            sq += v * v;
        }
        for (int i = threadIdx.x; i < Hkv * D; i += blockDim.x) {
            const float v = to_f32<T>(src[Hq * D + i]) + (bias ? bias[Hq * D + i] : 0.f);
            sk += v * v;
        }
        inv_q = 1.f / sqrtf(block_sum(sq, scratch) / (float)(Hq * D) + eps);
        if (Hkv > 0) inv_k = 1.f / sqrtf(block_sum(sk, scratch) / (float)(Hkv * D) + eps);
    }
    float* mine = head_s + (size_t)warp * 2 * D;
    float* turned = mine + D;
    for (int head = warp; head < Hq + Hkv; head += warps) {
        const T* x = src + (size_t)head * D;
        const float* b = bias ? bias + (size_t)head * D : nullptr;
        const float* w = head < Hq ? q_w : k_w;
        if (w && whole) w += (size_t)(head < Hq ? head : head - Hq) * D;      // weights over the whole projection
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) {
            const float v = to_f32<T>(x[d]) + (b ? b[d] : 0.f);
            mine[d] = v;
            ss += v * v;
        }
        if (normed && !after) {
            const float inv = whole ? (head < Hq ? inv_q : inv_k) : 1.f / sqrtf(warp_sum(ss) / (float)D + eps);
            for (int d = lane; d < D; d += 32) mine[d] = mine[d] * inv * (w ? w[d] : 1.f);
        }
        __syncwarp();
        ss = 0.f;
        for (int d = lane; d < D; d += 32) {
            float v = mine[d];
            if (d < 2 * rot_half) {
                const bool low = d < rot_half;
                const int t = low ? d : d - rot_half;
                const float p = mine[low ? d + rot_half : d - rot_half];
                v = low ? v * cr[t] - p * sr[t] : v * cr[t] + p * sr[t];
            }
            turned[d] = v;
            ss += v * v;
        }
        float inv = 1.f;
        if (normed && after) inv = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);       // per head: whole rows are normalised before
        T* dst = nullptr;
        if (head < Hq) dst = q_out + ((size_t)r * Hq + head) * Dk;
        else if (page_row >= 0) dst = k_pages + ((size_t)page_row + (size_t)(head - Hq) * page_size) * Dk;
        if (dst)
            for (int d = lane; d < Dk; d += 32) {                                    // each lane reads back what it wrote
                float v = d < D ? turned[d] : 0.f;
                if (normed && after && d < D) v = v * inv * (w ? w[d] : 1.f);
                if (head < Hq) v *= q_gain;
                dst[d] = from_f32<T>(v);
            }
        __syncwarp();
    }
    if (page_row >= 0 || mix_mode == QKV_MIX_SOURCE) {
        const T* v_src = src + (size_t)(Hq + Hkv) * D;
        const float* b = bias ? bias + (size_t)(Hq + Hkv) * D : nullptr;
        T* keep_row = kept ? kept + (size_t)r * Hkv * Dv : nullptr;
        for (int i = threadIdx.x; i < Hkv * Dv; i += blockDim.x) {
            const int hk = i / Dv, d = i - hk * Dv;
            float v = to_f32<T>(v_src[i]) + (b ? b[i] : 0.f);
            if (mix_mode == QKV_MIX_SOURCE) keep_row[i] = from_f32<T>(v);
            else if (mix_mode == QKV_MIX_BLEND) v = (1.f - mix) * v + mix * to_f32<T>(keep_row[i]);
            if (page_row >= 0) v_pages[((size_t)page_row + (size_t)hk * page_size) * Dvs + d] = from_f32<T>(v);
        }
        if (page_row >= 0 && Dvs > Dv)
            for (int i = threadIdx.x; i < Hkv * (Dvs - Dv); i += blockDim.x) {
                const int hk = i / (Dvs - Dv), d = Dv + i - hk * (Dvs - Dv);
                v_pages[((size_t)page_row + (size_t)hk * page_size) * Dvs + d] = from_f32<T>(0.f);
            }
    }
}

// The same for bfloat16 rows whose norm runs over the whole query (key) projection with weights, in steps of eight numbers:
// a block takes ROWS consecutive rows.  A thread reads 16 bytes at a time, adds the biases, leaves (x + b) * w in shared
// memory and its squares in two sums a row (queries, keys); after one barrier for the sums every thread takes chunks again,
// rotates them with their partner chunks from shared memory and multiplies by the row's inverse root mean square on the way
// out (the rotation is linear, so the order does not matter).  Values pass straight through.  What does not depend on the
// product before this kernel - positions, pages, angles, the first chunk's biases and weights - is fetched before the wait.
// A row's additions are the same whatever ROWS: the number of threads follows from the row's width alone.
template <int ROWS>
__global__ void __launch_bounds__(ROWS == 1 ? 1024 : 512)
qkv_whole_norm_rope_append_kernel(const bf16* __restrict__ qkv, int row_stride, const float* __restrict__ bias,
                                                  const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                                  const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_half,
                                                  int table_len, const int* __restrict__ positions, const int* __restrict__ row_segment,
                                                  const int* __restrict__ block_table, int table_stride, bf16* __restrict__ k_pages,
                                                  bf16* __restrict__ v_pages, bf16* __restrict__ q_out, int T, int Hq, int Hkv, int D,
                                                  int Dv, int Dk, int Dvs, int page_size, int write_kv, int* __restrict__ err) {
    extern __shared__ __align__(16) float row_s[];      // [ROWS][qk]: (x + b) * w, then [ROWS][2 rot_half]: cos, sin
    __shared__ float part_s[32][2 * ROWS];              // each warp's sums of squares
    __shared__ float inv_s[2 * ROWS];
    __shared__ long long page_row_s[ROWS];              // (page, slot) of the row's keys and values, counted in tokens; -1: none
    if (ROWS == 1) pdl_launch_dependents();             // a few small blocks: the successor may come onto the SMs at once
    const int r0 = blockIdx.x * ROWS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
    const int q_width = Hq * D, qk = (Hq + Hkv) * D, rot = 2 * rot_half;
    const int qk_chunks = qk >> 3, chunks = qk_chunks + (write_kv ? Hkv * Dv >> 3 : 0);
    float* angles = row_s + ROWS * qk;
    if (tid < ROWS) {
        const int r = r0 + tid;
        long long at = -1;
        if (r < T && write_kv) {
            const int pos = positions[r];
            const int page = block_table[(size_t)row_segment[r] * table_stride + pos / page_size];
            if (page < 0) atomicOr(err, KVB_DEV_BAD_PAGE);
            else at = (long long)page * Hkv * page_size + pos % page_size;
        }
        page_row_s[tid] = at;
    }
    for (int i = tid; i < ROWS * rot; i += blockDim.x) {
        const int row = i / rot, j = i - row * rot, r = r0 + row;
        float v = 0.f;
        if (r < T) {
            const int pos = positions[r];
            const bool pos_ok = pos >= 0 && pos < table_len;
            if (!pos_ok && j == 0) atomicOr(err, KVB_DEV_BAD_POS);
            const int p = pos_ok ? pos : 0;
            v = j < rot_half ? cos_t[(size_t)p * rot_half + j] : sin_t[(size_t)p * rot_half + j - rot_half];
        }
        angles[i] = v;
    }
    float b[8], w[8];
    auto constants = [&](int c) {                        // biases and weights of chunk c
        const int at = 8 * c;
        const float* ws = at < q_width ? q_w + at : k_w + at - q_width;
#pragma unroll
        for (int e = 0; e < 8; e += 4) {
            const float4 b4 = bias ? *reinterpret_cast<const float4*>(bias + at + e) : make_float4(0.f, 0.f, 0.f, 0.f);
            b[e] = b4.x; b[e + 1] = b4.y; b[e + 2] = b4.z; b[e + 3] = b4.w;
            const float4 w4 = c < qk_chunks ? *reinterpret_cast<const float4*>(ws + e) : make_float4(1.f, 1.f, 1.f, 1.f);
            w[e] = w4.x; w[e + 1] = w4.y; w[e + 2] = w4.z; w[e + 3] = w4.w;
        }
    };
    if (tid < chunks) constants(tid);
    pdl_wait();
    if (ROWS != 1) pdl_launch_dependents();
    __syncthreads();                                     // the rows' pages
    float sums[2 * ROWS];
#pragma unroll
    for (int i = 0; i < 2 * ROWS; ++i) sums[i] = 0.f;
    for (int c = tid; c < chunks; c += blockDim.x) {
        if (c != tid) constants(c);
        uint4 raw[ROWS];
#pragma unroll
        for (int row = 0; row < ROWS; ++row)
            raw[row] = *reinterpret_cast<const uint4*>(qkv + (size_t)min(r0 + row, T - 1) * row_stride + 8 * c);
#pragma unroll
        for (int row = 0; row < ROWS; ++row) {
            const uint32_t in[4] = {raw[row].x, raw[row].y, raw[row].z, raw[row].w};
            float x[8];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&in[k]));
                x[2 * k] = f.x + b[2 * k];
                x[2 * k + 1] = f.y + b[2 * k + 1];
            }
            if (c < qk_chunks) {
                float ss = 0.f;
#pragma unroll
                for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
                if (8 * c < q_width) sums[2 * row] += ss; else sums[2 * row + 1] += ss;
                float4* dst = reinterpret_cast<float4*>(row_s + row * qk + 8 * c);
                dst[0] = make_float4(x[0] * w[0], x[1] * w[1], x[2] * w[2], x[3] * w[3]);
                dst[1] = make_float4(x[4] * w[4], x[5] * w[5], x[6] * w[6], x[7] * w[7]);
            } else if (page_row_s[row] >= 0) {
                const int at = 8 * (c - qk_chunks), hk = at / Dv, d = at - hk * Dv;
                uint32_t o[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const __nv_bfloat162 v = __floats2bfloat162_rn(x[2 * k], x[2 * k + 1]);
                    o[k] = *reinterpret_cast<const uint32_t*>(&v);
                }
                *reinterpret_cast<uint4*>(v_pages + ((size_t)page_row_s[row] + (size_t)hk * page_size) * Dvs + d) = make_uint4(o[0], o[1], o[2], o[3]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2 * ROWS; ++i) {
        const float s = warp_sum(sums[i]);
        if (lane == 0) part_s[warp][i] = s;
    }
    __syncthreads();
    if (tid < 2 * ROWS) {
        float total = 0.f;
        for (int k = 0; k < warps; ++k) total += part_s[k][tid];
        const int n = (tid & 1) ? Hkv * D : q_width;
        inv_s[tid] = n > 0 ? 1.f / sqrtf(total / (float)n + eps) : 0.f;
    }
    __syncthreads();
    const int per_head = Dk >> 3;                        // chunks of a stored head: its own, then zeros
    for (int c = tid; c < (Hq + (write_kv ? Hkv : 0)) * per_head; c += blockDim.x) {
        const int head = c / per_head, d = 8 * (c - head * per_head);
        const bool is_q = head < Hq;
#pragma unroll
        for (int row = 0; row < ROWS; ++row) {
            if (r0 + row >= T || (!is_q && page_row_s[row] < 0)) continue;
            float x[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = 0.f;
            if (d < D) {
                const float* own = row_s + row * qk + head * D + d;
#pragma unroll
                for (int e = 0; e < 8; e += 4) {
                    const float4 v = *reinterpret_cast<const float4*>(own + e);
                    x[e] = v.x; x[e + 1] = v.y; x[e + 2] = v.z; x[e + 3] = v.w;
                }
                if (d < rot) {
                    const bool low = d < rot_half;
                    const float* partner = low ? own + rot_half : own - rot_half;
                    const float* cs = angles + row * rot + (low ? d : d - rot_half);
                    const float* sn = cs + rot_half;
#pragma unroll
                    for (int e = 0; e < 8; ++e) x[e] = low ? x[e] * cs[e] - partner[e] * sn[e] : x[e] * cs[e] + partner[e] * sn[e];
                }
                const float inv = inv_s[2 * row + (is_q ? 0 : 1)];
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] *= inv;
            }
            uint32_t o[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const __nv_bfloat162 v = __floats2bfloat162_rn(x[2 * k], x[2 * k + 1]);
                o[k] = *reinterpret_cast<const uint32_t*>(&v);
            }
            bf16* dst = is_q ? q_out + ((size_t)(r0 + row) * Hq + head) * Dk
                             : k_pages + ((size_t)page_row_s[row] + (size_t)(head - Hq) * page_size) * Dk;
            *reinterpret_cast<uint4*>(dst + d) = make_uint4(o[0], o[1], o[2], o[3]);
        }
    }
    if (write_kv && Dvs > Dv) {
        const int pad = (Dvs - Dv) >> 3;
        for (int i = tid; i < ROWS * Hkv * pad; i += blockDim.x) {
            const int row = i / (Hkv * pad), at = i - row * Hkv * pad, hk = at / pad, d = Dv + 8 * (at - hk * pad);
            if (page_row_s[row] >= 0)
                *reinterpret_cast<uint4*>(v_pages + ((size_t)page_row_s[row] + (size_t)hk * page_size) * Dvs + d) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
}

// KVB_ERR_LIMIT: sizes or addresses this kernel does not take (the caller has another).
static int launch_whole_norm(const bf16* qkv, int row_stride, const float* bias, const float* q_w, const float* k_w, float eps,
                             const float* cos_t, const float* sin_t, int rot_half, int table_len, const int* positions,
                             const int* row_segment, const int* block_table, int table_stride, bf16* k_pages, bf16* v_pages, bf16* q_out,
                             int T, int Hq, int Hkv, int D, int Dv, int Dk, int Dvs, int page_size, int write_kv, int* err,
                             cudaStream_t stream) {
    const uintptr_t addresses = (uintptr_t)qkv | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)q_out | (uintptr_t)bias | (uintptr_t)q_w | (uintptr_t)k_w;
    if ((addresses & 15) || ((row_stride | D | Dv | Dk | Dvs | rot_half) & 7)) return KVB_ERR_LIMIT;
    const int qk = (Hq + Hkv) * D;
    const int chunks = (qk + (write_kv ? Hkv * Dv : 0)) / 8;
    const int threads = chunks >= 1024 ? 1024 : (chunks + 31) / 32 * 32;
    constexpr int ROWS = 4;
    const size_t one = (size_t)(qk + 2 * rot_half) * sizeof(float);
    if (one > 46 * 1024) return KVB_ERR_LIMIT;           // 48 KB without an attribute, some of it the kernel's own
    if (T >= 256 && ROWS * one <= 46 * 1024 && threads <= 512)
        kvb_launch(qkv_whole_norm_rope_append_kernel<ROWS>, dim3((T + ROWS - 1) / ROWS), dim3(threads), ROWS * one, stream, qkv, row_stride,
                   bias, q_w, k_w, eps, cos_t, sin_t, rot_half, table_len, positions, row_segment, block_table, table_stride, k_pages,
                   v_pages, q_out, T, Hq, Hkv, D, Dv, Dk, Dvs, page_size, write_kv, err);
    else
        kvb_launch(qkv_whole_norm_rope_append_kernel<1>, dim3(T), dim3(threads), one, stream, qkv, row_stride, bias, q_w, k_w, eps, cos_t,
                   sin_t, rot_half, table_len, positions, row_segment, block_table, table_stride, k_pages, v_pages, q_out, T, Hq, Hkv, D,
                   Dv, Dk, Dvs, page_size, write_kv, err);
    return kvb_launch_status();
}

// `norm_flags`: QKV_NORM - queries and keys are normalised (weights q_w / k_w, or none); QKV_NORM_ALL - over a row's whole
// query (key) projection, all heads at once, with weights of that size, instead of per head with weights of D numbers
// that the heads share; QKV_NORM_AFTER - after the rotation instead of before it (per head only).  `mix_mode`:
// QKV_MIX_SOURCE - the row's values are also written to kept[r]; QKV_MIX_BLEND - v = (1 - lam[0]) v + lam[0] kept[r].
KVB_API int kvb_qkv_norm_rope_append(int dtype, const void* qkv, int row_stride, const float* bias, const float* q_w,
                                     const float* k_w, float eps, int norm_flags, const float* cos_t, const float* sin_t,
                                     int rot_half, int table_len, const int* positions, const int* row_segment,
                                     const int* block_table, int table_stride, void* k_pages, void* v_pages, void* q_out, int T,
                                     int Hq, int Hkv, int D, int Dv, int Dk, int page_size, int write_kv, int mix_mode, void* kept,
                                     const float* lam, int Dvs, float qt_coef, int qt_every, int* err, cudaStream_t stream) {
    if (T <= 0) return KVB_OK;
    if (2 * rot_half > D || rot_half < 0 || Dv < 1 || Dk < D || Dvs < Dv || qt_every < 0 || row_stride < (Hq + Hkv) * D + Hkv * Dv ||
        Hq < 1 || Hkv < 0 || (Hkv == 0 && (write_kv || mix_mode != 0)) || (Hkv > 0 && (q_w == nullptr) != (k_w == nullptr)))
        return KVB_ERR_SHAPE;
    if ((norm_flags & QKV_NORM_ALL) && (norm_flags & QKV_NORM_AFTER)) return KVB_ERR_SHAPE;
    if (mix_mode < 0 || mix_mode > QKV_MIX_BLEND || (mix_mode != 0 && kept == nullptr) || (mix_mode == QKV_MIX_BLEND && lam == nullptr))
        return KVB_ERR_SHAPE;
    if (dtype == KVB_BF16 && norm_flags == (QKV_NORM | QKV_NORM_ALL) && mix_mode == 0 && qt_every == 0 && q_w != nullptr) {
        const int rc = launch_whole_norm((const bf16*)qkv, row_stride, bias, q_w, k_w, eps, cos_t, sin_t, rot_half, table_len, positions,
                                         row_segment, block_table, table_stride, (bf16*)k_pages, (bf16*)v_pages, (bf16*)q_out, T, Hq, Hkv,
                                         D, Dv, Dk, Dvs, page_size, write_kv, err, stream);
        if (rc != KVB_ERR_LIMIT) return rc;
    }
    const int warps = Hq + Hkv >= 8 ? 8 : 4;
    const size_t smem = ((size_t)warps * 2 * D + 33) * sizeof(float);
    if (smem > 48 * 1024) return KVB_ERR_LIMIT;
    if (dtype == KVB_F32)
        kvb_launch(qkv_norm_rope_append_kernel<float>, dim3(T), dim3(32 * warps), smem, stream, (const float*)qkv, row_stride, bias,
                   q_w, k_w, eps, norm_flags, cos_t, sin_t, rot_half, table_len, positions, row_segment, block_table, table_stride,
                   (float*)k_pages, (float*)v_pages, (float*)q_out, Hq, Hkv, D, Dv, Dk, page_size, write_kv, mix_mode, (float*)kept,
                   lam, Dvs, qt_coef, qt_every, err);
    else if (dtype == KVB_BF16)
        kvb_launch(qkv_norm_rope_append_kernel<bf16>, dim3(T), dim3(32 * warps), smem, stream, (const bf16*)qkv, row_stride, bias,
                   q_w, k_w, eps, norm_flags, cos_t, sin_t, rot_half, table_len, positions, row_segment, block_table, table_stride,
                   (bf16*)k_pages, (bf16*)v_pages, (bf16*)q_out, Hq, Hkv, D, Dv, Dk, page_size, write_kv, mix_mode, (bf16*)kept,
                   lam, Dvs, qt_coef, qt_every, err);
    else
        return KVB_ERR_DTYPE;
    return kvb_launch_status();
}
