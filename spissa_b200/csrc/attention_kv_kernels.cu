// Causal grouped-query attention over the paged cache for bfloat16 keys and values of different sizes (or of a size that
// attention_kernels.cu is not built for): the kernels of flash_paged.cuh on tiles of 32, 64, 96 or 128 columns for keys and
// for values, whose rows may be any multiples of 8 up to the tiles'.
#include "flash_paged.cuh"

SP_API const char* sp_attention_kv_last_error() { return sp_error_text; }
SP_DEFINE_RANGE_API(attention_kv)

#define SP_KV_TILES(X) X(32, 32) X(32, 64) X(32, 96) X(32, 128) X(64, 32) X(64, 64) X(64, 96) X(64, 128) \
    X(96, 32) X(96, 64) X(96, 96) X(96, 128) X(128, 32) X(128, 64) X(128, 96) X(128, 128)

SP_API int sp_flash_kv_supported(int d, int vd, int nh, int nkv, int page_size) {
    return d >= 8 && d <= 128 && d % 8 == 0 && vd >= 8 && vd <= 128 && vd % 8 == 0 && nkv > 0 && nh % nkv == 0 && nh / nkv <= 16 && page_size == KT;
}

namespace {

int check_kv(int d, int vd, int nh, int nkv, int page_size, const void* q, const void* kpool, const void* vpool, const void* out) {
    if (!sp_flash_kv_supported(d, vd, nh, nkv, page_size))
        SP_FAIL("flash attention: keys of %d and values of %d (%d heads over %d, pages of %d) are not built", d, vd, nh, nkv, page_size);
    if (((uintptr_t)q | (uintptr_t)kpool | (uintptr_t)vpool | (uintptr_t)out) & 15) SP_FAIL("flash attention: operands must start on a 16-byte boundary");
    return 0;
}

template <int HD, int VD>
int launch_prefill(dim3 grid, cudaStream_t stream, const __nv_bfloat16* q, __nv_bfloat16* out, const PagedKV& kv, const int* seq_start,
                   const int* positions, int n_seqs, int nh, int window, float sl, int d, int vd) {
    static SpPerDevice ok;
    if (!ok.done()) { if (opt_in_smem(flash_prefill_kernel<HD, VD, true>, prefill_smem<HD, VD>(), "flash_prefill")) return 1; ok.mark(); }
    SP_CHECK_CALL("flash_prefill (kv)", sp_launch_dependent(flash_prefill_kernel<HD, VD, true>, grid, dim3(128), (size_t)prefill_smem<HD, VD>(), stream,
                                                            q, out, kv, seq_start, positions, n_seqs, nh, window, sl, d, vd));
    return 0;
}

template <int HD, int VD, int NH>
int launch_decode(dim3 grid, cudaStream_t stream, const __nv_bfloat16* q, const PagedKV& kv, const int* seq_len, int nh, int window,
                  float sl, int chunk_tiles, float* part_o, float* part_ml, int* counters, void* out, int out_dt, int d, int vd) {
    static SpPerDevice ok;
    if (!ok.done()) { if (opt_in_smem(flash_decode_kernel<HD, NH, VD, true>, decode_smem<HD, VD>(), "flash_decode")) return 1; ok.mark(); }
    SP_CHECK_CALL("flash_decode (kv)", sp_launch_dependent(flash_decode_kernel<HD, NH, VD, true>, grid, dim3(128), (size_t)decode_smem<HD, VD>(), stream,
                                                           q, kv, seq_len, nh, window, sl, chunk_tiles, part_o, part_ml, counters, out, out_dt, d, vd));
    return 0;
}

int tile_of(int n) { return (n + 31) / 32 * 32; }

}  // namespace

// as sp_flash_prefill, with key rows of ``d`` and value rows of ``vd``; out [T, nh*vd]
SP_API int sp_flash_prefill_kv(const void* q, void* out, const void* kpool, const void* vpool, const int* seq_start,
                               const int* positions, const int* seq_row, const int* page_table, int max_pages, int page_size,
                               int n_seqs, int n_q_tiles, int nh, int nkv, int d, int vd, int window, float scale,
                               const float* sink, const float* dist_bias, int dist_cap, cudaStream_t stream) {
    if (n_q_tiles <= 0) return 0;
    if (check_kv(d, vd, nh, nkv, page_size, q, kpool, vpool, out)) return 1;
    if (dist_bias && dist_cap < 0) SP_FAIL("flash_prefill: a distance-bias table needs at least one entry per head");
    if (n_q_tiles > 65535) SP_FAIL("flash_prefill: %d query tiles are beyond this kernel's grid", n_q_tiles);
    PagedKV kv{(const __nv_bfloat16*)kpool, (const __nv_bfloat16*)vpool, page_table, seq_row, max_pages, nkv, sp_range_host, sink,
               dist_bias, dist_cap};
    const dim3 grid(nh, n_q_tiles);
    const int th = tile_of(d), tv = tile_of(vd);
#define X(a, b) if (th == a && tv == b) return launch_prefill<a, b>(grid, stream, (const __nv_bfloat16*)q, (__nv_bfloat16*)out, kv, seq_start, positions, n_seqs, nh, window, scale * LOG2E, d, vd);
    SP_KV_TILES(X)
#undef X
    SP_FAIL("flash_prefill: tiles of %d and %d are not built", th, tv);
}

// as sp_flash_decode; scratch: n_seqs*nh*n_chunks*(vd + 2) floats
SP_API int sp_flash_decode_kv(const void* q, void* out, int out_dt, const void* kpool, const void* vpool, const int* seq_len,
                              const int* seq_row, const int* page_table, int max_pages, int page_size, int n_seqs, int nh, int nkv,
                              int d, int vd, int window, float scale, int chunk_tiles, int n_chunks, float* scratch,
                              long long scratch_floats, int* counters, const float* sink, const float* dist_bias, int dist_cap,
                              cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (check_kv(d, vd, nh, nkv, page_size, q, kpool, vpool, out)) return 1;
    if (dist_bias && dist_cap < 0) SP_FAIL("flash decode: a distance-bias table needs at least one entry per head");
    if (chunk_tiles <= 0 || n_chunks <= 0 || n_chunks > 65535 || n_seqs > 65535) SP_FAIL("flash decode: bad chunking %d x %d of %d sequences", n_chunks, chunk_tiles, n_seqs);
    const long long need = (long long)n_seqs * nh * n_chunks * (vd + 2);
    if (scratch_floats < need) SP_FAIL("flash decode: scratch holds %lld floats, %lld are needed", scratch_floats, need);
    PagedKV kv{(const __nv_bfloat16*)kpool, (const __nv_bfloat16*)vpool, page_table, seq_row, max_pages, nkv, sp_range_host, sink,
               dist_bias, dist_cap};
    float* part_o = scratch;
    float* part_ml = scratch + (size_t)n_seqs * nh * n_chunks * vd;
    const dim3 grid(n_chunks, nkv, n_seqs);
    const int th = tile_of(d), tv = tile_of(vd);
    const bool one = nh <= 8 * nkv;
    int rc = -1;
#define X(a, b) if (th == a && tv == b) rc = one ? launch_decode<a, b, 1>(grid, stream, (const __nv_bfloat16*)q, kv, seq_len, nh, window, scale * LOG2E, chunk_tiles, part_o, part_ml, counters, out, out_dt, d, vd) \
                                                 : launch_decode<a, b, 2>(grid, stream, (const __nv_bfloat16*)q, kv, seq_len, nh, window, scale * LOG2E, chunk_tiles, part_o, part_ml, counters, out, out_dt, d, vd);
    SP_KV_TILES(X)
#undef X
    if (rc < 0) SP_FAIL("flash decode: tiles of %d and %d are not built", th, tv);
    if (rc) return rc;
    if (counters) return 0;                  // the last CTA of every (sequence, kv head) has combined
    if (out_dt == SP_DT_BF16)
        decode_combine_kernel<__nv_bfloat16><<<n_seqs * nh, 128, 0, stream>>>(part_o, part_ml, (__nv_bfloat16*)out, n_chunks, vd, sink, nh);
    else
        decode_combine_kernel<float><<<n_seqs * nh, 128, 0, stream>>>(part_o, part_ml, (float*)out, n_chunks, vd, sink, nh);
    SP_CHECK_LAUNCH("decode_combine");
    return 0;
}
