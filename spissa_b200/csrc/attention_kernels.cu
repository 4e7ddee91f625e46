// Causal grouped-query attention over the paged cache for bfloat16 storage: a prefill kernel
// (many query tokens per sequence) and a decode kernel (one query token per sequence, keys
// split over CTAs, then combined).
//
// Meaning as in the reference (crates/spissa-runtime/src/rotary.rs:335-415, softmax :549-569):
// score = q·k / sqrt(head_dim); keys after the query are not seen (nor keys before
// pos-window+1 when a window is set); softmax in 32-bit with the maximum subtracted;
// output = sum p·v; query head h reads kv head h / (heads / kv_heads).
//
// Both kernels walk the keys in tiles of 64 = one cache page ([page][kv head][64][head_dim],
// so a tile is one contiguous block), staged in shared memory with cp.async, double
// buffered. Products run on mma.sync m16n8k16 (bfloat16 in, float32 out); the running
// maximum, sum and output stay in float32 registers (online softmax in the log2 domain).
// Prefill: a CTA owns 64 consecutive query tokens of one head; each of its 4 warps owns 16.
// Decode: a CTA owns the query heads of one kv head of one sequence (as the 16 rows of one
// tile, unused rows zero) for one chunk of key tiles; each warp takes 16 keys of every tile.
// Keys that no query may see are masked whatever the cache holds there; the cache is
// zero-initialised so that a masked weight of zero never meets a NaN value.
#include "flash_paged.cuh"

SP_API const char* sp_attention_last_error() { return sp_error_text; }
SP_DEFINE_RANGE_API(attention)

namespace {

// Head sizes the kernels are instantiated for: every multiple of 16 up to 128 (the fragments of mma.sync are 16 wide;
// beyond 128 a thread's output row no longer fits its registers and the generic kernel runs).
#define SP_FLASH_HEAD_SIZES(X) X(16) X(32) X(48) X(64) X(80) X(96) X(112) X(128)

bool head_size_built(int hd) { return hd >= 16 && hd <= 128 && hd % 16 == 0; }

int check_common(int hd, int nh, int nkv, int page_size) {
    if (!head_size_built(hd)) SP_FAIL("flash attention: head_dim %d is not built (multiples of 16 up to 128 are)", hd);
    if (nkv <= 0 || nh % nkv) SP_FAIL("flash attention: %d heads are no multiple of %d kv heads", nh, nkv);
    if (page_size != KT) SP_FAIL("flash attention: pages of %d tokens, this kernel walks pages of %d", page_size, KT);
    return 0;
}

}  // namespace

// Whether the flash kernels are built for this shape (1) or the generic kernel has to run (0).
// Query rows per CTA of the prefill kernel (= the page size its key tiles have): the host counts tiles with it.
SP_API int sp_flash_query_tile() { return KT; }

SP_API int sp_flash_supported(int hd, int nh, int nkv, int page_size) {
    return head_size_built(hd) && nkv > 0 && nh % nkv == 0 && nh / nkv <= 16 && page_size == KT;
}

namespace {
template <int HD>
int launch_flash_prefill_as(dim3 grid, cudaStream_t stream, const __nv_bfloat16* q, __nv_bfloat16* out, const PagedKV& kv,
                            const int* seq_start, const int* positions, int n_seqs, int nh, int window, float sl) {
    static SpPerDevice ok;            // the opt-in holds for one device: asked for on each device's first launch
    if (!ok.done()) { if (opt_in_smem(flash_prefill_kernel<HD>, prefill_smem<HD>(), "flash_prefill")) return 1; ok.mark(); }
    sp_launch_dependent(flash_prefill_kernel<HD>, grid, dim3(128), (size_t)prefill_smem<HD>(), stream, q, out, kv, seq_start,
                        positions, n_seqs, nh, window, sl, HD, HD);
    return 0;
}
}  // namespace

// ``sink`` (float32 per query head, or null): a score that joins every row's denominator once, with no key and no value
// ``dist_bias`` (float32 [nh][dist_cap + 1], or null): a score added by the distance between query and key
SP_API int sp_flash_prefill_bias(const void* q, void* out, const void* kpool, const void* vpool, const int* seq_start,
                                 const int* positions, const int* seq_row, const int* page_table, int max_pages,
                                 int page_size, int n_seqs, int n_q_tiles, int nh, int nkv, int hd, int window,
                                 float scale, const float* sink, const float* dist_bias, int dist_cap, cudaStream_t stream) {
    if (n_q_tiles <= 0) return 0;
    if (check_common(hd, nh, nkv, page_size)) return 1;
    if (dist_bias && dist_cap < 0) SP_FAIL("flash_prefill: a distance-bias table needs at least one entry per head");
    PagedKV kv{(const __nv_bfloat16*)kpool, (const __nv_bfloat16*)vpool, page_table, seq_row, max_pages, nkv, sp_range_host, sink,
               dist_bias, dist_cap};
    if (n_q_tiles > 65535) SP_FAIL("flash_prefill: %d query tiles are beyond this kernel's grid", n_q_tiles);
    dim3 grid(nh, n_q_tiles);
    const float sl = scale * LOG2E;
    switch (hd) {
#define X(n)                                                                                                        \
    case n:                                                                                                         \
        if (launch_flash_prefill_as<n>(grid, stream, (const __nv_bfloat16*)q, (__nv_bfloat16*)out, kv, seq_start,   \
                                       positions, n_seqs, nh, window, sl)) return 1;                                \
        break;
        SP_FLASH_HEAD_SIZES(X)
#undef X
    }
    SP_CHECK_LAUNCH("flash_prefill");
    return 0;
}

SP_API int sp_flash_prefill_sink(const void* q, void* out, const void* kpool, const void* vpool, const int* seq_start,
                                 const int* positions, const int* seq_row, const int* page_table, int max_pages,
                                 int page_size, int n_seqs, int n_q_tiles, int nh, int nkv, int hd, int window,
                                 float scale, const float* sink, cudaStream_t stream) {
    return sp_flash_prefill_bias(q, out, kpool, vpool, seq_start, positions, seq_row, page_table, max_pages, page_size,
                                 n_seqs, n_q_tiles, nh, nkv, hd, window, scale, sink, nullptr, 0, stream);
}

SP_API int sp_flash_prefill(const void* q, void* out, const void* kpool, const void* vpool, const int* seq_start,
                            const int* positions, const int* seq_row, const int* page_table, int max_pages,
                            int page_size, int n_seqs, int n_q_tiles, int nh, int nkv, int hd, int window,
                            float scale, cudaStream_t stream) {
    return sp_flash_prefill_sink(q, out, kpool, vpool, seq_start, positions, seq_row, page_table, max_pages, page_size,
                                 n_seqs, n_q_tiles, nh, nkv, hd, window, scale, nullptr, stream);
}

namespace {
// One instantiation per head size and number of head tiles (query heads per kv head: up to 8, up to 16).
template <int HD, int NH>
int launch_flash_decode_as(dim3 grid, cudaStream_t stream, const __nv_bfloat16* q, const PagedKV& kv, const int* seq_len,
                           int nh, int window, float sl, int chunk_tiles, float* part_o, float* part_ml, int* counters,
                           void* out, int out_dt) {
    static SpPerDevice ok;            // the opt-in holds for one device: asked for on each device's first launch
    if (!ok.done()) { if (opt_in_smem(flash_decode_kernel<HD, NH>, decode_smem<HD>(), "flash_decode")) return 1; ok.mark(); }
    sp_launch_dependent(flash_decode_kernel<HD, NH>, grid, dim3(128), (size_t)decode_smem<HD>(), stream, q, kv, seq_len, nh, window, sl,
                        chunk_tiles, part_o, part_ml, counters, out, out_dt, HD, HD);
    return 0;
}
int launch_flash_decode(int hd, dim3 grid, cudaStream_t stream, const __nv_bfloat16* q, const PagedKV& kv,
                        const int* seq_len, int nh, int window, float sl, int chunk_tiles, float* part_o, float* part_ml,
                        int* counters, void* out, int out_dt) {
    const bool one = nh <= 8 * kv.nkv;
    switch (hd) {
#define X(n)                                                                                                              \
    case n:                                                                                                               \
        return one ? launch_flash_decode_as<n, 1>(grid, stream, q, kv, seq_len, nh, window, sl, chunk_tiles, part_o, part_ml, counters, out, out_dt) \
                   : launch_flash_decode_as<n, 2>(grid, stream, q, kv, seq_len, nh, window, sl, chunk_tiles, part_o, part_ml, counters, out, out_dt);
        SP_FLASH_HEAD_SIZES(X)
#undef X
    }
    SP_FAIL("flash decode: head_dim %d is not built", hd);
}

}  // namespace

// Floats of scratch the decode kernels need: part_o then part_ml. ``counters`` (optional, n_seqs·nkv ints,
// zero before the first launch; the kernel returns them to zero) lets the last CTA combine the chunks;
// without it a second kernel does.
SP_API long long sp_flash_decode_scratch_floats(int n_seqs, int nh, int hd, int n_chunks) {
    return (long long)n_seqs * nh * n_chunks * (hd + 2);
}

SP_API int sp_flash_decode_bias(const void* q, void* out, int out_dt, const void* kpool, const void* vpool,
                                const int* seq_len, const int* seq_row, const int* page_table, int max_pages,
                                int page_size, int n_seqs, int nh, int nkv, int hd, int window, float scale,
                                int chunk_tiles, int n_chunks, float* scratch, long long scratch_floats, int* counters,
                                const float* sink, const float* dist_bias, int dist_cap, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (check_common(hd, nh, nkv, page_size)) return 1;
    if (dist_bias && dist_cap < 0) SP_FAIL("flash decode: a distance-bias table needs at least one entry per head");
    if (nh / nkv > 16) SP_FAIL("flash decode: %d query heads per kv head, at most 16 fit one tile", nh / nkv);
    if (chunk_tiles <= 0 || n_chunks <= 0 || n_chunks > 65535) SP_FAIL("flash decode: bad chunking %d x %d", n_chunks, chunk_tiles);
    if (n_seqs > 65535) SP_FAIL("flash decode: %d sequences are beyond this kernel's grid", n_seqs);
    const long long need = sp_flash_decode_scratch_floats(n_seqs, nh, hd, n_chunks);
    if (scratch_floats < need) SP_FAIL("flash decode: scratch holds %lld floats, %lld are needed", scratch_floats, need);
    PagedKV kv{(const __nv_bfloat16*)kpool, (const __nv_bfloat16*)vpool, page_table, seq_row, max_pages, nkv, sp_range_host, sink,
               dist_bias, dist_cap};
    float* part_o = scratch;
    float* part_ml = scratch + (size_t)n_seqs * nh * n_chunks * hd;
    dim3 grid(n_chunks, nkv, n_seqs);
    const float sl = scale * LOG2E;
    if (launch_flash_decode(hd, grid, stream, (const __nv_bfloat16*)q, kv, seq_len, nh, window, sl, chunk_tiles, part_o,
                            part_ml, counters, out, out_dt)) return 1;
    SP_CHECK_LAUNCH("flash_decode");
    if (counters) return 0;                  // the last CTA of every (sequence, kv head) has combined
    if (out_dt == SP_DT_BF16)
        decode_combine_kernel<__nv_bfloat16><<<n_seqs * nh, hd <= 64 ? 64 : 128, 0, stream>>>(part_o, part_ml, (__nv_bfloat16*)out, n_chunks, hd, sink, nh);
    else
        decode_combine_kernel<float><<<n_seqs * nh, hd <= 64 ? 64 : 128, 0, stream>>>(part_o, part_ml, (float*)out, n_chunks, hd, sink, nh);
    SP_CHECK_LAUNCH("decode_combine");
    return 0;
}

SP_API int sp_flash_decode_sink(const void* q, void* out, int out_dt, const void* kpool, const void* vpool,
                                const int* seq_len, const int* seq_row, const int* page_table, int max_pages,
                                int page_size, int n_seqs, int nh, int nkv, int hd, int window, float scale,
                                int chunk_tiles, int n_chunks, float* scratch, long long scratch_floats, int* counters,
                                const float* sink, cudaStream_t stream) {
    return sp_flash_decode_bias(q, out, out_dt, kpool, vpool, seq_len, seq_row, page_table, max_pages, page_size, n_seqs, nh,
                                nkv, hd, window, scale, chunk_tiles, n_chunks, scratch, scratch_floats, counters, sink, nullptr, 0,
                                stream);
}

SP_API int sp_flash_decode(const void* q, void* out, int out_dt, const void* kpool, const void* vpool,
                           const int* seq_len, const int* seq_row, const int* page_table, int max_pages,
                           int page_size, int n_seqs, int nh, int nkv, int hd, int window, float scale,
                           int chunk_tiles, int n_chunks, float* scratch, long long scratch_floats, int* counters,
                           cudaStream_t stream) {
    return sp_flash_decode_sink(q, out, out_dt, kpool, vpool, seq_len, seq_row, page_table, max_pages, page_size, n_seqs, nh,
                                nkv, hd, window, scale, chunk_tiles, n_chunks, scratch, scratch_floats, counters, nullptr, stream);
}

// ------------------------------------------------------------------ decode without a caller's scratch
// See attention_noalloc.h. The scratch of the split-key decode kernel lives here, in the library.
#include "attention_noalloc.h"

static __device__ __align__(256) float sp_static_partials[SP_FLASH_DECODE_STATIC_MAX_FLOATS];
static __device__ __align__(256) int sp_static_counters[SP_FLASH_DECODE_STATIC_MAX_COUNTERS];

namespace {
constexpr int STATIC_MAX_DEVICES = 64;
float* static_partials_ptr[STATIC_MAX_DEVICES];      // device addresses, looked up once per device
int* static_counters_ptr[STATIC_MAX_DEVICES];
}  // namespace

SP_API int sp_flash_decode_static(const void* q, void* out, int out_dt, const void* kpool, const void* vpool,
                                  const int* seq_len, const int* seq_row, const int* page_table, int max_pages,
                                  int page_size, int n_seqs, int nh, int nkv, int hd, int window, float scale,
                                  int chunk_tiles, int n_chunks, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (check_common(hd, nh, nkv, page_size)) return 1;
    if (nh / nkv > 16) SP_FAIL("flash decode: %d query heads per kv head, at most 16 fit one tile", nh / nkv);
    if (chunk_tiles <= 0 || n_chunks <= 0 || n_chunks > 65535) SP_FAIL("flash decode: bad chunking %d x %d", n_chunks, chunk_tiles);
    if (n_seqs > 65535) SP_FAIL("flash decode: %d sequences are beyond this kernel's grid", n_seqs);
    if (out_dt != SP_DT_F32 && out_dt != SP_DT_BF16) SP_FAIL("flash decode: unsupported output dtype code %d", out_dt);
    const long long need = sp_flash_decode_scratch_floats(n_seqs, nh, hd, n_chunks);
    if (need > (long long)SP_FLASH_DECODE_STATIC_MAX_FLOATS)
        SP_FAIL("flash decode (static scratch): %lld floats of partial results are needed, the built-in array holds %d; "
                "use fewer chunks or the entry point that takes a scratch buffer", need, SP_FLASH_DECODE_STATIC_MAX_FLOATS);
    if ((long long)n_seqs * nkv > (long long)SP_FLASH_DECODE_STATIC_MAX_COUNTERS)
        SP_FAIL("flash decode (static scratch): %lld arrival counters are needed, the built-in array holds %d",
                (long long)n_seqs * nkv, SP_FLASH_DECODE_STATIC_MAX_COUNTERS);

    // the arrays' names are host-side handles; kernels need their device addresses, per device
    int dev = -1;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) SP_FAIL("flash decode (static scratch): cudaGetDevice failed: %s", cudaGetErrorString(e));
    if (dev < 0 || dev >= STATIC_MAX_DEVICES) SP_FAIL("flash decode (static scratch): device %d is beyond the %d this build tracks", dev, STATIC_MAX_DEVICES);
    if (!static_partials_ptr[dev]) {
        float* pp = nullptr;
        int* cp = nullptr;
        e = cudaGetSymbolAddress((void**)&pp, sp_static_partials);
        if (e != cudaSuccess || !pp) SP_FAIL("flash decode (static scratch): no address for the partial-result array: %s", cudaGetErrorString(e));
        e = cudaGetSymbolAddress((void**)&cp, sp_static_counters);
        if (e != cudaSuccess || !cp) SP_FAIL("flash decode (static scratch): no address for the counter array: %s", cudaGetErrorString(e));
        static_counters_ptr[dev] = cp;
        static_partials_ptr[dev] = pp;
    }
    float* part_o = static_partials_ptr[dev];
    float* part_ml = part_o + (size_t)n_seqs * nh * n_chunks * hd;
    int* counters = static_counters_ptr[dev];
    // the counters must start at zero whatever an earlier, perhaps interrupted, call left there
    e = cudaMemsetAsync(counters, 0, (size_t)n_seqs * nkv * sizeof(int), stream);
    if (e != cudaSuccess) SP_FAIL("flash decode (static scratch): clearing the counters failed: %s", cudaGetErrorString(e));

    PagedKV kv{(const __nv_bfloat16*)kpool, (const __nv_bfloat16*)vpool, page_table, seq_row, max_pages, nkv, sp_range_host};
    dim3 grid(n_chunks, nkv, n_seqs);
    const float sl = scale * LOG2E;
    if (launch_flash_decode(hd, grid, stream, (const __nv_bfloat16*)q, kv, seq_len, nh, window, sl, chunk_tiles, part_o,
                            part_ml, counters, out, out_dt)) return 1;
    SP_CHECK_LAUNCH("flash_decode (static scratch)");
    return 0;
}
