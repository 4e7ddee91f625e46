// The paged attention kernels of attention_kernels.cu (keys and values of one size) and attention_kv_kernels.cu (sizes of
// their own): a prefill kernel, a decode kernel with split keys, its combining pass.
#pragma once
#include "flash_common.cuh"

namespace {

constexpr int DEC_STAGES = 3;                 // tiles in flight per warp of the decode kernel

// Rows of keys and values need not have one size, nor one that a kernel is built for: HD and VD are the sizes of the
// shared-memory tiles, d and vd (multiples of 8) those of the rows; with PAD they may be smaller, and what the tiles hold
// the query and key tiles hold beyond them is zero (a value tile's columns beyond vd lead to outputs that nobody stores).
__device__ __forceinline__ void zero_columns(uint32_t tile, int rows, int row_bytes, int from, int to, int tid, int nthreads) {
    const int n = (to - from) / 8;                    // 16-byte pieces
    for (int c = tid; c < rows * n; c += nthreads)
        asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(tile + (c / n) * row_bytes + from * 2 + (c % n) * 16), "r"(0u) : "memory");
}

// ------------------------------------------------------------------ prefill
template <int HD, int VD = HD, bool PAD = false>
__global__ void __launch_bounds__(128)
flash_prefill_kernel(const __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ out, PagedKV kv,
                     const int* __restrict__ seq_start, const int* __restrict__ positions, int n_seqs, int nh,
                     int window, float scale_log2, int d_ = HD, int vd_ = VD) {
    using T = Tile<HD>;
    using TV = Tile<VD>;
    const int d = PAD ? d_ : HD, vd = PAD ? vd_ : VD;
    extern __shared__ __align__(128) uint8_t smem[];
    const uint32_t q_tile = smem_u32(smem);
    const uint32_t k_tiles = q_tile + T::BYTES;          // two stages of K, then two of V
    const uint32_t v_tiles = k_tiles + 2 * T::BYTES;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    sp_allow_dependents();
    sp_wait_for_predecessor();

    // which sequence and which 64-token tile of it. Heads run fastest over the grid and tiles from the last to the
    // first: the tiles with the most keys start first in every head, the short ones fill the end.
    int x = (int)gridDim.y - 1 - (int)blockIdx.y, b = 0, first = 0, n_new = 0;
    for (; b < n_seqs; ++b) {
        first = seq_start[b];
        n_new = seq_start[b + 1] - first;
        const int nt = (n_new + KT - 1) / KT;
        if (x < nt) break;
        x -= nt;
    }
    if (b >= n_seqs) return;
    const int t0 = first + x * KT;
    const int n_rows = min(KT, n_new - x * KT);
    const int pos0 = positions[t0];
    const int h = blockIdx.x;
    const int g = h / (nh / kv.nkv);
    const int* pt = kv.page_table + (size_t)sp_checked_row(kv.seq_row[b], kv.rg) * kv.max_pages;

    const int last_pos = pos0 + n_rows - 1;
    const int first_key = (window > 0 && pos0 - window + 1 > 0) ? pos0 - window + 1 : 0;
    const int j_lo = first_key / KT, j_hi = last_pos / KT;

    if (PAD && d < HD) {
        zero_columns(q_tile, 3 * KT, T::ROW, d, HD, tid, 128);      // the queries and both stages of keys
        __syncthreads();
    }
    load_tile_async<HD>(q_tile, q + (size_t)t0 * nh * d + (size_t)h * d, (size_t)nh * d, n_rows, tid, 128, d);
    {
        const size_t off = ((size_t)sp_checked_page(pt[sp_checked_entry(j_lo, kv.max_pages, kv.rg)], kv.rg) * kv.nkv + g) * KT;
        load_tile_async<HD>(k_tiles, kv.k + off * d, d, KT, tid, 128, d);
        load_tile_async<VD>(v_tiles, kv.v + off * vd, vd, KT, tid, 128, vd);
    }
    cp_async_commit();

    uint32_t qf[HD / 16][4];
    float o[VD / 8][4];
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    const int r0 = warp * 16 + (lane >> 2);
    const int hi[2] = {pos0 + r0, pos0 + r0 + 8};
    const int lo[2] = {window > 0 ? hi[0] - window + 1 : 0, window > 0 ? hi[1] - window + 1 : 0};
    const int warp_hi = pos0 + warp * 16 + 15;                     // last key any row of this warp may see
    const int warp_lo = window > 0 ? pos0 + warp * 16 - window + 1 : 0;
    const bool warp_active = warp * 16 < n_rows;
    const float* bias_row = kv.dist_bias ? kv.dist_bias + (size_t)h * (kv.dist_cap + 1) : nullptr;

    for (int j = j_lo; j <= j_hi; ++j) {
        const int stage = (j - j_lo) & 1;
        if (j < j_hi) {
            const size_t off = ((size_t)sp_checked_page(pt[sp_checked_entry(j + 1, kv.max_pages, kv.rg)], kv.rg) * kv.nkv + g) * KT;
            load_tile_async<HD>(k_tiles + (stage ^ 1) * T::BYTES, kv.k + off * d, d, KT, tid, 128, d);
            load_tile_async<VD>(v_tiles + (stage ^ 1) * TV::BYTES, kv.v + off * vd, vd, KT, tid, 128, vd);
        }
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        if (j == j_lo) load_q_frags<HD>(q_tile, warp * 16, lane, qf);
        const int tile_pos0 = j * KT;
        if (warp_active && tile_pos0 <= warp_hi && tile_pos0 + KT - 1 >= warp_lo) {
            // every key of the tile is at or before the warp's first row and inside its last row's window
            const bool all_seen = tile_pos0 + KT - 1 <= pos0 + warp * 16 && (window <= 0 || tile_pos0 >= warp_hi - window + 1);
            if (all_seen)
                flash_step<HD, 8, false, VD>(qf, k_tiles + stage * T::BYTES, v_tiles + stage * TV::BYTES, 0, tile_pos0, lo, hi,
                                         scale_log2, o, m, l, lane, bias_row, kv.dist_cap);
            else
                flash_step<HD, 8, true, VD>(qf, k_tiles + stage * T::BYTES, v_tiles + stage * TV::BYTES, 0, tile_pos0, lo, hi,
                                        scale_log2, o, m, l, lane, bias_row, kv.dist_cap);
        }
        __syncthreads();
    }
    cp_async_wait<0>();

#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    }
    if (kv.sink) {
        const float sk = kv.sink[h] * LOG2E;           // the row's maximum m is in log2 units
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float m_all = fmaxf(m[r], sk), f = exp2f(m[r] - m_all);
            l[r] = l[r] * f + exp2f(sk - m_all);
#pragma unroll
            for (int i = 0; i < VD / 8; ++i) { o[i][2 * r] *= f; o[i][2 * r + 1] *= f; }
        }
    }
    const int t = lane & 3;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = warp * 16 + (lane >> 2) + r * 8;
        if (row >= n_rows) continue;
        const float inv = 1.0f / l[r];
        __nv_bfloat16* dst = out + (size_t)(t0 + row) * nh * vd + (size_t)h * vd;
#pragma unroll
        for (int i = 0; i < VD / 8; ++i)
            if (!PAD || i * 8 < vd) *(uint32_t*)(dst + i * 8 + 2 * t) = pack_bf16(o[i][2 * r] * inv, o[i][2 * r + 1] * inv);
    }
}

// The CTA that finishes last for a (sequence, kv head) combines all chunks of its G heads, in chunk
// order whatever the order of arrival, and hands the counter back at zero for the next launch.
template <int VD>
__device__ __forceinline__ void combine_if_last(const float* part_o, const float* part_ml, int* counters, void* out,
                                                int out_dt, int b, int g, int G, int nh, int nkv, int n_chunks,
                                                int* is_last, const float* sink = nullptr, int vd = VD) {
    __threadfence();                                    // this CTA's partials are visible before it is counted
    __syncthreads();
    if (threadIdx.x == 0) {
        const int prev = atomicAdd(&counters[b * nkv + g], 1);
        *is_last = (prev == n_chunks - 1);
        if (*is_last) counters[b * nkv + g] = 0;
    }
    __syncthreads();
    if (!*is_last) return;
    __threadfence();
    for (int e = threadIdx.x; e < G * vd; e += blockDim.x) {
        const int row = e / vd, d = e % vd;
        const size_t bh = (size_t)b * nh + (size_t)g * G + row;
        float mm = -INFINITY;
        for (int c = 0; c < n_chunks; ++c) mm = fmaxf(mm, __ldcg(&part_ml[(bh * n_chunks + c) * 2]));
        const float sk = sink ? sink[(size_t)g * G + row] * LOG2E : -INFINITY;
        mm = fmaxf(mm, sk);
        const float msafe = (mm == -INFINITY) ? 0.0f : mm;
        float ll = sink ? exp2f(sk - msafe) : 0.0f, acc = 0.0f;
        for (int c = 0; c < n_chunks; ++c) {
            const float lc = __ldcg(&part_ml[(bh * n_chunks + c) * 2 + 1]);
            if (lc > 0.0f) {
                const float f = exp2f(__ldcg(&part_ml[(bh * n_chunks + c) * 2]) - msafe);
                ll += lc * f;
                acc += __ldcg(&part_o[(bh * n_chunks + c) * vd + d]) * f;
            }
        }
        sp_st_dt(out, out_dt, bh * vd + d, acc / ll);
    }
}

// ------------------------------------------------------------------ decode
// grid (chunks, kv heads, sequences). part_o [B][nh][chunks][HD], part_ml [B][nh][chunks][2] (m in log2 units).
template <int HD, int NH, int VD = HD, bool PAD = false>
__global__ void __launch_bounds__(128)
flash_decode_kernel(const __nv_bfloat16* __restrict__ q, PagedKV kv, const int* __restrict__ seq_len, int nh,
                    int window, float scale_log2, int chunk_tiles, float* __restrict__ part_o,
                    float* __restrict__ part_ml, int* __restrict__ counters, void* __restrict__ out, int out_dt,
                    int d_ = HD, int vd_ = VD) {
    using T = Tile<HD>;
    using TV = Tile<VD>;
    const int d = PAD ? d_ : HD, vd = PAD ? vd_ : VD;
    extern __shared__ __align__(128) uint8_t smem[];
    const uint32_t q_tile = smem_u32(smem);                       // 16 rows used
    const uint32_t k_tiles = q_tile + 16 * T::ROW;
    const uint32_t v_tiles = k_tiles + DEC_STAGES * T::BYTES;
    float* merge = (float*)(smem + 16 * T::ROW + DEC_STAGES * (T::BYTES + TV::BYTES));    // [4 warps][16 rows][VD + 2]
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int chunk = blockIdx.x, n_chunks = gridDim.x, g = blockIdx.y, b = blockIdx.z;
    const int G = nh / kv.nkv;
    const int p = seq_len[b] - 1;                                  // the query's position
    const int first_key = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
    const int j_first = first_key / KT + chunk * chunk_tiles;
    const int j_last = min(p / KT, j_first + chunk_tiles - 1);
    const size_t part_base = ((size_t)b * nh + (size_t)g * G) * n_chunks + chunk;   // + head_in_group * n_chunks

    __shared__ int is_last;
    if (j_first > j_last) {                                        // nothing for this chunk
        for (int i = tid; i < G; i += 128) {
            part_ml[(part_base + (size_t)i * n_chunks) * 2] = -INFINITY;
            part_ml[(part_base + (size_t)i * n_chunks) * 2 + 1] = 0.0f;
        }
        if (counters) combine_if_last<VD>(part_o, part_ml, counters, out, out_dt, b, g, G, nh, kv.nkv, n_chunks, &is_last, kv.sink, vd);
        return;
    }
    const int* pt = kv.page_table + (size_t)sp_checked_row(kv.seq_row[b], kv.rg) * kv.max_pages;

    if (PAD && d < HD) {
        zero_columns(q_tile, 16 + DEC_STAGES * KT, T::ROW, d, HD, tid, 128);      // the queries and all stages of keys
        __syncthreads();
    }
    // the G heads of this kv head as rows 0..G-1 of a 16-row tile
    for (int c = tid; c < 16 * T::CHUNKS; c += 128) {
        const int r = c / T::CHUNKS, k = c % T::CHUNKS;
        const uint32_t to = q_tile + r * T::ROW + k * 16;
        if (PAD && k * 8 >= d) continue;
        if (r < G) cp_async16(to, q + (size_t)b * nh * d + (size_t)(g * G + r) * d + k * 8);
        else asm volatile("st.shared.v4.b32 [%0], {%1,%1,%1,%1};" ::"r"(to), "r"(0u) : "memory");
    }
    cp_async_commit();                                             // group 0: the queries

    // keys are the M of the products, the group's heads their N, in NH tiles of 8 (decode_step_t)
    uint32_t qb[HD / 16][NH][2];
    float o[VD / 16][NH][4], m[NH][2], l[NH][2];
#pragma unroll
    for (int i = 0; i < NH; ++i) {
        m[i][0] = m[i][1] = -INFINITY;
        l[i][0] = l[i][1] = 0.0f;
#pragma unroll
        for (int dt = 0; dt < VD / 16; ++dt) o[dt][i][0] = o[dt][i][1] = o[dt][i][2] = o[dt][i][3] = 0.0f;
    }

    // Each warp fetches and uses only its own 16 keys of every tile, so inside the loop the warps
    // need no barrier among themselves: a warp waits for its own copies and goes on.
    auto fetch = [&](int j, int stage) {
        const size_t off = ((size_t)sp_checked_page(pt[sp_checked_entry(j, kv.max_pages, kv.rg)], kv.rg) * kv.nkv + g) * KT + (size_t)warp * 16;
        const uint32_t kt = k_tiles + stage * T::BYTES + warp * 16 * T::ROW;
        const uint32_t vt = v_tiles + stage * TV::BYTES + warp * 16 * TV::ROW;
        if (HD == VD && !PAD) {
            for (int c = lane; c < 16 * T::CHUNKS; c += 32) {
                const int r = c / T::CHUNKS, k = c % T::CHUNKS;
                cp_async16(kt + r * T::ROW + k * 16, kv.k + (off + r) * HD + k * 8);
                cp_async16(vt + r * T::ROW + k * 16, kv.v + (off + r) * HD + k * 8);
            }
        } else {
            for (int c = lane; c < 16 * T::CHUNKS; c += 32) {
                const int r = c / T::CHUNKS, k = c % T::CHUNKS;
                if (k * 8 < d) cp_async16(kt + r * T::ROW + k * 16, kv.k + (off + r) * d + k * 8);
            }
            for (int c = lane; c < 16 * TV::CHUNKS; c += 32) {
                const int r = c / TV::CHUNKS, k = c % TV::CHUNKS;
                if (k * 8 < vd) cp_async16(vt + r * TV::ROW + k * 16, kv.v + (off + r) * vd + k * 8);
            }
        }
    };
#pragma unroll
    for (int s = 0; s < DEC_STAGES - 1; ++s) {
        if (j_first + s <= j_last) fetch(j_first + s, s);
        cp_async_commit();
    }
    cp_async_wait<DEC_STAGES - 1>();                               // the queries have landed (all later groups may fly)
    __syncthreads();
    // Qᵀ as the B operand: lane (g, t) holds dims 2t, 2t+1 and 2t+8, 2t+9 of head g of each head tile
#pragma unroll
    for (int kk = 0; kk < HD / 16; ++kk)
#pragma unroll
        for (int i = 0; i < NH; ++i) {
            const uint32_t a = q_tile + (i * 8 + (lane >> 2)) * T::ROW + (kk * 16 + 2 * (lane & 3)) * 2;
            asm volatile("ld.shared.b32 %0, [%1];" : "=r"(qb[kk][i][0]) : "r"(a));
            asm volatile("ld.shared.b32 %0, [%1];" : "=r"(qb[kk][i][1]) : "r"(a + 16));
        }

    const float* bias_group = kv.dist_bias ? kv.dist_bias + (size_t)g * G * (kv.dist_cap + 1) : nullptr;
    for (int j = j_first; j <= j_last; ++j) {
        const int it = j - j_first;
        const int stage = it % DEC_STAGES;
        if (j + DEC_STAGES - 1 <= j_last) fetch(j + DEC_STAGES - 1, (it + DEC_STAGES - 1) % DEC_STAGES);
        cp_async_commit();
        cp_async_wait<DEC_STAGES - 1>();
        __syncwarp();
        if (j * KT + KT - 1 <= p && j * KT >= first_key)
            decode_step_t<HD, NH, false, VD>(qb, k_tiles + stage * T::BYTES, v_tiles + stage * TV::BYTES, warp * 16, j * KT,
                                         first_key, p, scale_log2, o, m, l, lane, bias_group, kv.dist_cap, G);
        else
            decode_step_t<HD, NH, true, VD>(qb, k_tiles + stage * T::BYTES, v_tiles + stage * TV::BYTES, warp * 16, j * KT,
                                        first_key, p, scale_log2, o, m, l, lane, bias_group, kv.dist_cap, G);
        __syncwarp();                                              // the stage is free for this warp's next fetch
    }
    cp_async_wait<0>();

    // merge the four warps' (m, l, o): each covered other keys of the same rows
    constexpr int MS = VD + 2;
    const int lg = lane >> 2, lt = lane & 3;
#pragma unroll
    for (int i = 0; i < NH; ++i)
#pragma unroll
        for (int c = 0; c < 2; ++c) {                              // head 8i + 2·lt + c: dims lg and lg + 8 of every 16
            l[i][c] += __shfl_xor_sync(0xffffffffu, l[i][c], 4);   // the lanes that share lt hold the head's other keys
            l[i][c] += __shfl_xor_sync(0xffffffffu, l[i][c], 8);
            l[i][c] += __shfl_xor_sync(0xffffffffu, l[i][c], 16);
            float* dst = merge + ((size_t)warp * 16 + i * 8 + 2 * lt + c) * MS;
#pragma unroll
            for (int dt = 0; dt < VD / 16; ++dt) {
                dst[dt * 16 + lg] = o[dt][i][c];
                dst[dt * 16 + lg + 8] = o[dt][i][c + 2];
            }
            if (lg == 0) { dst[VD] = m[i][c]; dst[VD + 1] = l[i][c]; }
        }
    __syncthreads();
    for (int e = tid; e < G * vd; e += 128) {
        const int row = e / vd, c = e % vd;
        float mm = -INFINITY;
#pragma unroll
        for (int w = 0; w < 4; ++w) mm = fmaxf(mm, merge[((size_t)w * 16 + row) * MS + VD]);
        const float msafe = (mm == -INFINITY) ? 0.0f : mm;
        float acc = 0.0f, ll = 0.0f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float* src = merge + ((size_t)w * 16 + row) * MS;
            const float f = exp2f(src[VD] - msafe);
            acc += src[c] * f;
            ll += src[VD + 1] * f;
        }
        const size_t pi = part_base + (size_t)row * n_chunks;
        part_o[pi * vd + c] = acc;
        if (c == 0) { part_ml[pi * 2] = mm; part_ml[pi * 2 + 1] = ll; }
    }
    if (counters) combine_if_last<VD>(part_o, part_ml, counters, out, out_dt, b, g, G, nh, kv.nkv, n_chunks, &is_last, kv.sink, vd);
}

// out[b, head, :] = sum_c o_c·2^(m_c - M) / sum_c l_c·2^(m_c - M), chunks in order
template <typename TO>
__global__ void decode_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                      TO* __restrict__ out, int n_chunks, int HD, const float* __restrict__ sink, int nh) {
    const size_t bh = blockIdx.x;
    float mm = -INFINITY;
    for (int c = 0; c < n_chunks; ++c) mm = fmaxf(mm, part_ml[(bh * n_chunks + c) * 2]);
    const float sk = sink ? sink[bh % nh] * LOG2E : -INFINITY;
    mm = fmaxf(mm, sk);
    const float msafe = (mm == -INFINITY) ? 0.0f : mm;
    float ll = sink ? exp2f(sk - msafe) : 0.0f;
    for (int c = 0; c < n_chunks; ++c)
        ll += part_ml[(bh * n_chunks + c) * 2 + 1] * exp2f(part_ml[(bh * n_chunks + c) * 2] - msafe);
    const float inv = 1.0f / ll;
    for (int d = threadIdx.x; d < HD; d += blockDim.x) {
        float acc = 0.0f;
        for (int c = 0; c < n_chunks; ++c) {
            const float lc = part_ml[(bh * n_chunks + c) * 2 + 1];
            if (lc > 0.0f) acc += part_o[(bh * n_chunks + c) * HD + d] * exp2f(part_ml[(bh * n_chunks + c) * 2] - msafe);
        }
        sp_st(out, bh * HD + d, acc * inv);
    }
}

template <int HD, int VD = HD>
constexpr int prefill_smem() { return 3 * Tile<HD>::BYTES + 2 * Tile<VD>::BYTES; }
template <int HD, int VD = HD>
constexpr int decode_smem() { return 16 * Tile<HD>::ROW + DEC_STAGES * (Tile<HD>::BYTES + Tile<VD>::BYTES) + 4 * 16 * (VD + 2) * 4; }

template <typename Kern>
int opt_in_smem(Kern kern, int bytes, const char* name) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) SP_FAIL("%s: cannot reserve %d bytes of shared memory: %s", name, bytes, cudaGetErrorString(e));
    return 0;
}

}  // namespace
