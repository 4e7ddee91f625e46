// Small kernels of layers whose sublayers stand between two norms, and of gated attention mixers.
//
//   pair_embed          x_t = s · E[id_t] + B[(id_{t−1} · a + id_t · b) mod n]; the first token of a sequence takes the
//                       table's row n. The token before a step's first one is a word of per-slot state.
//   stream_norm_add     x ← x + r · y / sqrt(mean(y²) + eps) ⊙ w for a sublayer's output y (which is left zeroed for
//                       the next sublayer to add into); in the same pass the next reader's input: the norm of the new
//                       x with another weight, or the new x as it is, in the activation type; ``centered``: both norms
//                       are layer norms (mean taken off, a weight, no bias)
//   gated_qkv_store     a projected row [q | k | v | one gate per head]: biases, a query factor that grows with the
//                       logarithm of the position, rotation of neighbouring pairs over the first dims of every head,
//                       q out, k and v into their page rows, the gates out as 32-bit numbers
//   qkv_norm_rot_store  a projected row [q | k | v]: biases, an RMS norm with a weight of every q and k head, rotation of
//                       pairs half the rotated dims apart (or neighbouring ones), q out, k and v into their page rows
//   latent_rot_store    a projected row [q (per head: plain | rotated part) | low-rank row | shared key part | gates]:
//                       RMS norm of the low-rank row, rotation of the shared key part and of the queries' rotated
//                       parts (neighbouring dims or dims half the part apart form a pair), [normed row | rotated key
//                       part] into ONE page row, q and the gates out
//   gelu_gather_mul     out[t, j] = gelu_tanh(z[t, j]) · S[id_t, off + j]
//
// Norm statistics, angles (position · frequency, cosf / sinf), gates and sums are 32-bit; stores round to the
// activation type.
#include "common.cuh"

SP_API const char* sp_sandwich_last_error() { return sp_error_text; }
SP_DEFINE_RANGE_API(sandwich)

// ============================================================== token row plus pair row
struct PairEmbedArgs {
    const void* table; const void* pairs; int dt;   // [vocab][W], [buckets + 1][W]
    const int* ids; const int* positions; const int* token_seq; const int* seq_start; const int* seq_slot;
    int* state; int n_slots;                        // [slots]: the last token of the step before
    float* out;
    int T, W, vocab, buckets, mul_prev, mul_cur;
    float scale;
    int* status;
};

__global__ void __launch_bounds__(128) pair_embed_kernel(PairEmbedArgs a) {
    __shared__ int row_s;
    const int t = blockIdx.x;
    if (t >= a.T) return;
    const int id = a.ids[t];
    const bool ok = id >= 0 && id < a.vocab;
    if (threadIdx.x == 0) {
        const int s = a.token_seq[t], first = a.seq_start[s];
        int slot = a.seq_slot[s];
        if (slot < 0 || slot >= a.n_slots) slot = 0;
        int row = a.buckets;                                        // a sequence's first token: the last row
        if (a.positions[t] > 0) {
            const int prev = t > first ? a.ids[t - 1] : a.state[slot];
            const long long mix = (long long)prev * a.mul_prev + (long long)id * a.mul_cur;
            row = (int)(((mix % a.buckets) + a.buckets) % a.buckets);
        }
        row_s = row;
        // the block of a sequence's first token of the step has read the state; it leaves the step's last token there
        if (t == first) a.state[slot] = a.ids[a.seq_start[s + 1] - 1];
        if (!ok && a.status) atomicCAS(a.status, 0, 301);           // a token id outside the table
    }
    __syncthreads();
    const int row = row_s;
    for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
        const float e = ok ? sp_ld_dt(a.table, a.dt, (size_t)id * a.W + c) * a.scale : 0.0f;
        a.out[(size_t)t * a.W + c] = ok ? e + sp_ld_dt(a.pairs, a.dt, (size_t)row * a.W + c) : 0.0f;
    }
}

SP_API int sp_pair_embed(const void* table, const void* pairs, int dt, const int* ids, const int* positions,
                         const int* token_seq, const int* seq_start, const int* seq_slot, int* state, int n_slots, float* out,
                         int T, int W, int vocab, int buckets, int mul_prev, int mul_cur, float scale, int* status,
                         cudaStream_t stream) {
    if (T <= 0) return 0;
    if (buckets <= 0) SP_FAIL("pair_embed: the pair table needs at least one bucket, got %d", buckets);
    PairEmbedArgs a{table, pairs, dt, ids, positions, token_seq, seq_start, seq_slot, state, n_slots, out,
                    T, W, vocab, buckets, mul_prev, mul_cur, scale, status};
    pair_embed_kernel<<<T, 128, 0, stream>>>(a);
    SP_CHECK_LAUNCH("pair_embed");
    return 0;
}

// ============================================================== norm of a sublayer's output into the stream
struct NormAddArgs {
    float* x; float* y;                  // [T][W] the stream; the sublayer's output (zeroed on the way out)
    const float* w_post;                 // [W] weight of the output's norm, as it multiplies
    const float* w_next;                 // [W] weight of the next reader's norm, or null
    void* out; int out_dt;               // [T][W] the next reader's input, or null
    int next_mode;                       // 0: no output; 1: norm of the new x with w_next; 2: the new x as it is
    int T, W;
    float mult, eps;
};

template <int VEC>
__global__ void __launch_bounds__(256) stream_norm_add_kernel(NormAddArgs a) {
    __shared__ float red[32];
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int t = blockIdx.x;
    if (t >= a.T) return;
    float* xr = a.x + (size_t)t * a.W;
    float* yr = a.y + (size_t)t * a.W;
    float ss = 0.0f;
    if (VEC == 4) {
        for (int c = threadIdx.x * 4; c < a.W; c += blockDim.x * 4) {
            const float4 v = *(const float4*)(yr + c);
            ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
        }
    } else {
        for (int c = threadIdx.x; c < a.W; c += blockDim.x) ss = fmaf(yr[c], yr[c], ss);
    }
    ss = sp_block_sum(ss, red);
    const float f = a.mult / sqrtf(ss / (float)a.W + a.eps);
    float s2 = 0.0f;
    if (VEC == 4) {
        for (int c = threadIdx.x * 4; c < a.W; c += blockDim.x * 4) {
            const float4 v = *(const float4*)(yr + c), w = *(const float4*)(a.w_post + c);
            float4 x = *(const float4*)(xr + c);
            x.x = fmaf(v.x * f, w.x, x.x); x.y = fmaf(v.y * f, w.y, x.y); x.z = fmaf(v.z * f, w.z, x.z); x.w = fmaf(v.w * f, w.w, x.w);
            *(float4*)(xr + c) = x;
            *(float4*)(yr + c) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            s2 = fmaf(x.x, x.x, s2); s2 = fmaf(x.y, x.y, s2); s2 = fmaf(x.z, x.z, s2); s2 = fmaf(x.w, x.w, s2);
        }
    } else {
        for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
            const float x = fmaf(yr[c] * f, a.w_post[c], xr[c]);
            xr[c] = x;
            yr[c] = 0.0f;
            s2 = fmaf(x, x, s2);
        }
    }
    if (a.next_mode == 0) return;
    float g = 1.0f;
    if (a.next_mode == 1) {
        s2 = sp_block_sum(s2, red);
        g = 1.0f / sqrtf(s2 / (float)a.W + a.eps);
    }
    // every thread reads back the entries it wrote itself
    if (VEC == 4) {
        for (int c = threadIdx.x * 4; c < a.W; c += blockDim.x * 4) {
            float4 x = *(const float4*)(xr + c);
            if (a.next_mode == 1) {
                const float4 w = *(const float4*)(a.w_next + c);
                x.x *= g * w.x; x.y *= g * w.y; x.z *= g * w.z; x.w *= g * w.w;
            }
            if (a.out_dt == SP_DT_F32) {
                *(float4*)((float*)a.out + (size_t)t * a.W + c) = x;
            } else {
                __nv_bfloat162 p0 = __floats2bfloat162_rn(x.x, x.y), p1 = __floats2bfloat162_rn(x.z, x.w);
                uint2 pk;
                pk.x = *(uint32_t*)&p0; pk.y = *(uint32_t*)&p1;
                *(uint2*)((__nv_bfloat16*)a.out + (size_t)t * a.W + c) = pk;
            }
        }
    } else {
        for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
            float x = xr[c];
            if (a.next_mode == 1) x *= g * a.w_next[c];
            sp_st_dt(a.out, a.out_dt, (size_t)t * a.W + c, x);
        }
    }
}

// The same with layer norms: (v − mean) / sqrt(mean((v − mean)²) + eps) ⊙ w for the output and for the next reader.
// Widths of 512 · NV: a block of 128 threads per row, the row in registers, mean and squared deviations of equal parts merged
// pair by pair (each part's are its own, so nothing cancels): one exchange through shared memory per norm.
struct MeanDev { float mean, dev; };              // of n numbers: their mean, the sum of their squared deviations from it
__device__ __forceinline__ MeanDev merge_equal(MeanDev a, MeanDev b, float n) {      // n: numbers in each part
    const float d = b.mean - a.mean;
    return MeanDev{0.5f * (a.mean + b.mean), a.dev + b.dev + 0.5f * n * d * d};
}
template <int N>
__device__ __forceinline__ MeanDev block_mean_dev(const float4 (&v)[N], MeanDev* red) {
    float s = 0.0f;
#pragma unroll
    for (int i = 0; i < N; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    MeanDev m{s * (1.0f / (4 * N)), 0.0f};
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const float p = v[i].x - m.mean, q = v[i].y - m.mean, r = v[i].z - m.mean, u = v[i].w - m.mean;
        m.dev += (p * p + q * q) + (r * r + u * u);
    }
    float n = 4.0f * N;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1, n *= 2.0f)
        m = merge_equal(m, MeanDev{__shfl_xor_sync(0xffffffffu, m.mean, o), __shfl_xor_sync(0xffffffffu, m.dev, o)}, n);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = m;
    __syncthreads();
    return merge_equal(merge_equal(red[0], red[1], n), merge_equal(red[2], red[3], n), 2.0f * n);
}

template <int NV>
__global__ void __launch_bounds__(128) stream_layernorm_add_rows_kernel(NormAddArgs a) {
    __shared__ MeanDev red[2][4];
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int t = blockIdx.x;
    if (t >= a.T) return;
    float4* __restrict__ xr = (float4*)(a.x + (size_t)t * a.W) + threadIdx.x;
    float4* __restrict__ yr = (float4*)(a.y + (size_t)t * a.W) + threadIdx.x;
    const float4* __restrict__ w1 = (const float4*)a.w_post + threadIdx.x;
    float4 v[NV], x[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) v[i] = yr[128 * i];
#pragma unroll
    for (int i = 0; i < NV; ++i) x[i] = xr[128 * i];
    const float invW = 1.0f / (float)a.W;
    const MeanDev m = block_mean_dev<NV>(v, red[0]);
    const float f = a.mult / sqrtf(m.dev * invW + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const float4 w = __ldg(w1 + 128 * i);
        x[i].x = fmaf((v[i].x - m.mean) * f, w.x, x[i].x); x[i].y = fmaf((v[i].y - m.mean) * f, w.y, x[i].y);
        x[i].z = fmaf((v[i].z - m.mean) * f, w.z, x[i].z); x[i].w = fmaf((v[i].w - m.mean) * f, w.w, x[i].w);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        xr[128 * i] = x[i];
        yr[128 * i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    if (a.next_mode == 0) return;
    MeanDev m2{0.0f, 0.0f};
    float g = 1.0f;
    if (a.next_mode == 1) {
        m2 = block_mean_dev<NV>(x, red[1]);
        g = 1.0f / sqrtf(m2.dev * invW + a.eps);
    }
    const float4* __restrict__ w2 = (const float4*)a.w_next + threadIdx.x;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        float4 o = x[i];
        if (a.next_mode == 1) {
            const float4 w = __ldg(w2 + 128 * i);
            o.x = (o.x - m2.mean) * g * w.x; o.y = (o.y - m2.mean) * g * w.y; o.z = (o.z - m2.mean) * g * w.z; o.w = (o.w - m2.mean) * g * w.w;
        }
        const size_t at = (size_t)t * a.W + (threadIdx.x + 128 * i) * 4;
        if (a.out_dt == SP_DT_F32) {
            *(float4*)((float*)a.out + at) = o;
        } else {
            __nv_bfloat162 p0 = __floats2bfloat162_rn(o.x, o.y), p1 = __floats2bfloat162_rn(o.z, o.w);
            uint2 pk;
            pk.x = *(uint32_t*)&p0; pk.y = *(uint32_t*)&p1;
            *(uint2*)((__nv_bfloat16*)a.out + at) = pk;
        }
    }
}

// any width: the mean first, then the squared deviations
__global__ void __launch_bounds__(256) stream_layernorm_add_kernel(NormAddArgs a) {
    __shared__ float red[32];
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int t = blockIdx.x;
    if (t >= a.T) return;
    float* xr = a.x + (size_t)t * a.W;
    float* yr = a.y + (size_t)t * a.W;
    const float invW = 1.0f / (float)a.W;
    float sum = 0.0f, ss = 0.0f;
    for (int c = threadIdx.x; c < a.W; c += blockDim.x) sum += yr[c];
    const float mean = sp_block_sum(sum, red) * invW;
    for (int c = threadIdx.x; c < a.W; c += blockDim.x) { const float v = yr[c] - mean; ss = fmaf(v, v, ss); }
    const float f = a.mult / sqrtf(sp_block_sum(ss, red) * invW + a.eps);
    sum = 0.0f;
    for (int c = threadIdx.x; c < a.W; c += blockDim.x) {
        const float x = fmaf((yr[c] - mean) * f, a.w_post[c], xr[c]);
        xr[c] = x;
        yr[c] = 0.0f;
        sum += x;
    }
    if (a.next_mode == 0) return;
    float m2 = 0.0f, g = 1.0f;
    if (a.next_mode == 1) {
        m2 = sp_block_sum(sum, red) * invW;
        ss = 0.0f;
        for (int c = threadIdx.x; c < a.W; c += blockDim.x) { const float v = xr[c] - m2; ss = fmaf(v, v, ss); }
        g = 1.0f / sqrtf(sp_block_sum(ss, red) * invW + a.eps);
    }
    for (int c = threadIdx.x; c < a.W; c += blockDim.x)
        sp_st_dt(a.out, a.out_dt, (size_t)t * a.W + c, a.next_mode == 1 ? (xr[c] - m2) * g * a.w_next[c] : xr[c]);
}

SP_API int sp_stream_norm_add(float* x, float* y, const float* w_post, const float* w_next, void* out, int out_dt,
                              int next_mode, int T, int W, float mult, float eps, int centered, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (next_mode < 0 || next_mode > 2 || (next_mode && !out) || (next_mode == 1 && !w_next))
        SP_FAIL("stream_norm_add: mode %d needs an output (and a weight for the norm)", next_mode);
    NormAddArgs a{x, y, w_post, w_next, out, out_dt, next_mode, T, W, mult, eps};
    const bool vec = (W % 4) == 0 && ((((uintptr_t)x | (uintptr_t)y | (uintptr_t)w_post | (uintptr_t)w_next | (uintptr_t)out) & 15) == 0);
    if (centered) {
#define SP_LN_ROWS(NV) if (vec && W == 512 * NV) { SP_CHECK_CALL("stream_norm_add", sp_launch_dependent(stream_layernorm_add_rows_kernel<NV>, dim3(T), dim3(128), 0, stream, a)); return 0; }
        SP_LN_ROWS(1) SP_LN_ROWS(2) SP_LN_ROWS(3) SP_LN_ROWS(4) SP_LN_ROWS(5) SP_LN_ROWS(6) SP_LN_ROWS(8) SP_LN_ROWS(10)
#undef SP_LN_ROWS
        SP_CHECK_CALL("stream_norm_add", sp_launch_dependent(stream_layernorm_add_kernel, dim3(T), dim3(256), 0, stream, a));
        return 0;
    }
    if (vec) SP_CHECK_CALL("stream_norm_add", sp_launch_dependent(stream_norm_add_kernel<4>, dim3(T), dim3(256), 0, stream, a));
    else SP_CHECK_CALL("stream_norm_add", sp_launch_dependent(stream_norm_add_kernel<1>, dim3(T), dim3(256), 0, stream, a));
    return 0;
}

// ============================================================== where a token's cached rows live
struct RowPlace {
    const int* token_seq; const int* positions; const int* seq_row; const int* page_table;
    int max_pages, page_size;
    SpRange rg;
};

__device__ __forceinline__ bool page_of(const RowPlace& pl, int t, int pos, int& page) {
    const int row = pl.seq_row[pl.token_seq[t]];
    if (!sp_index_ok(row, pl.rg.n_rows, pl.rg, 402) || !sp_index_ok(pos / pl.page_size, pl.max_pages, pl.rg, 403)) return false;
    page = pl.page_table[(size_t)row * pl.max_pages + pos / pl.page_size];
    return sp_index_ok(page, pl.rg.n_pages, pl.rg, 401);
}

// cos and sin of position · freq[i], times ``mult``, for i < half: cs[i], cs[half + i]
__device__ __forceinline__ void pair_angles(float* cs, const float* __restrict__ freq, int half, int pos, float mult) {
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float ang = (float)pos * freq[i];
        cs[i] = cosf(ang) * mult;
        cs[half + i] = sinf(ang) * mult;
    }
}

// ============================================================== [q | k | v | gates]: bias, query factor, rotation, store
struct GatedQkvArgs {
    const float* proj; int ld;           // [T][ld] = [q: nh·d | k: nkv·d | v: nkv·vd | gates: nh]
    const void* bias; int b_dt;          // [nh·d + nkv·d + nkv·vd] or null
    void* q_out; int q_dt;               // [T][nh·d]
    void* kpool; void* vpool; int c_dt;  // [pages][nkv][page_size][d], [pages][nkv][page_size][vd]
    float* gates;                        // [T][nh] the gates' arguments (their sigmoid is taken where they multiply)
    const float* freq;                   // [rd/2] or null
    RowPlace pl;
    int T, nh, nkv, d, vd, rd, write_kv;
    float rot_mult;                      // multiplies cos and sin
    float temp_coef; int temp_every;     // q ← q · (1 + coef · ln(floor((pos + 1) / every) + 1)); coef 0: no factor
};

template <typename TO, typename TC>
__global__ void __launch_bounds__(128) gated_qkv_store_kernel(GatedQkvArgs a) {
    extern __shared__ float cs[];        // [2][rd/2]
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int t = blockIdx.x;
    if (t >= a.T) return;
    const int pos = a.pl.positions[t];
    const int half = a.rd >> 1;
    pair_angles(cs, a.freq, half, pos, a.rot_mult);
    __syncthreads();
    int page = 0;
    const bool place_ok = a.write_kv && page_of(a.pl, t, pos, page);
    const int off = pos % a.pl.page_size;
    const float* src = a.proj + (size_t)t * a.ld;
    const float temp = a.temp_coef != 0.0f
        ? 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every) + 1.0f) : 1.0f;       // the quotient of integers: exact
    TO* q_out = (TO*)a.q_out;
    TC* kpool = (TC*)a.kpool;
    TC* vpool = (TC*)a.vpool;
    const int d = a.d, nq = a.nh, nqk = a.nh + a.nkv;
    if ((d & 1) == 0) {
        const int dp = d >> 1;
        for (int e = threadIdx.x; e < nqk * dp; e += blockDim.x) {
            const int h = e / dp, i = e - h * dp;
            const int c = h * d + 2 * i;
            float u = src[c], v = src[c + 1];
            if (a.bias) { u += sp_ld_dt(a.bias, a.b_dt, c); v += sp_ld_dt(a.bias, a.b_dt, c + 1); }
            if (h < nq) { u *= temp; v *= temp; }
            if (2 * i < a.rd) {
                const float co = cs[i], si = cs[half + i];
                const float ru = u * co - v * si, rv = v * co + u * si;
                u = ru; v = rv;
            }
            if (h < nq) sp_st2(q_out, (size_t)t * nq * d + c, u, v);
            else if (place_ok) sp_st2(kpool, (((size_t)page * a.nkv + (h - nq)) * a.pl.page_size + off) * d + 2 * i, u, v);
        }
    } else {
        // an odd head size: element by element; rd is even, so the last dim never turns
        for (int e = threadIdx.x; e < nqk * d; e += blockDim.x) {
            const int h = e / d, i = e - h * d;
            float val = src[e] + (a.bias ? sp_ld_dt(a.bias, a.b_dt, e) : 0.0f);
            if (i < a.rd) {
                const int im = i ^ 1;
                const float other = src[h * d + im] + (a.bias ? sp_ld_dt(a.bias, a.b_dt, h * d + im) : 0.0f);
                const float co = cs[i >> 1], si = cs[half + (i >> 1)];
                val = (i & 1) ? val * co + other * si : val * co - other * si;
            }
            if (h < nq) sp_st(q_out, (size_t)t * nq * d + e, val * temp);
            else if (place_ok) sp_st(kpool, (((size_t)page * a.nkv + (h - nq)) * a.pl.page_size + off) * d + i, val);
        }
    }
    const int v0 = nqk * d;
    if (place_ok) {
        for (int e = threadIdx.x; e < a.nkv * a.vd; e += blockDim.x) {
            const int g = e / a.vd, r = e - g * a.vd;
            float v = src[v0 + e];
            if (a.bias) v += sp_ld_dt(a.bias, a.b_dt, v0 + e);
            sp_st(vpool, (((size_t)page * a.nkv + g) * a.pl.page_size + off) * a.vd + r, v);
        }
    }
    if (a.gates) {
        const int g0 = v0 + a.nkv * a.vd;
        for (int h = threadIdx.x; h < a.nh; h += blockDim.x) a.gates[(size_t)t * a.nh + h] = src[g0 + h];
    }
}

SP_API int sp_gated_qkv_store(const float* proj, int ld, const void* bias, int b_dt, void* q_out, int q_dt, void* kpool,
                              void* vpool, int c_dt, float* gates, const float* freq, const int* token_seq,
                              const int* positions, const int* seq_row, const int* page_table, int max_pages, int page_size,
                              int T, int nh, int nkv, int d, int vd, int rd, int write_kv, float rot_mult, float temp_coef,
                              int temp_every, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || vd <= 0 || rd < 0 || rd > d || (rd & 1)) SP_FAIL("gated_qkv_store: the rotated dims %d must be even and at most %d", rd, d);
    if (rd > 0 && !freq) SP_FAIL("gated_qkv_store: a frequency table is needed");
    if (temp_coef != 0.0f && temp_every <= 0) SP_FAIL("gated_qkv_store: the query factor's period must be positive, got %d", temp_every);
    if (ld < (nh + nkv) * d + nkv * vd + (gates ? nh : 0)) SP_FAIL("gated_qkv_store: rows of %d numbers are too short", ld);
    GatedQkvArgs a{proj, ld, bias, b_dt, q_out, q_dt, kpool, vpool, c_dt, gates, freq,
                   RowPlace{token_seq, positions, seq_row, page_table, max_pages, page_size, sp_range_host},
                   T, nh, nkv, d, vd, rd, write_kv, rot_mult, temp_coef, temp_every};
    const size_t smem = (size_t)(rd > 0 ? rd : 2) * sizeof(float);
#define GQ_LAUNCH(TO, TC) SP_CHECK_CALL("gated_qkv_store", sp_launch_dependent(gated_qkv_store_kernel<TO, TC>, dim3(T), dim3(128), smem, stream, a))
    if (q_dt == SP_DT_F32 && c_dt == SP_DT_F32) GQ_LAUNCH(float, float);
    else if (q_dt == SP_DT_BF16 && c_dt == SP_DT_BF16) GQ_LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else if (q_dt == SP_DT_F32 && c_dt == SP_DT_BF16) GQ_LAUNCH(float, __nv_bfloat16);
    else if (q_dt == SP_DT_BF16 && c_dt == SP_DT_F32) GQ_LAUNCH(__nv_bfloat16, float);
    else SP_FAIL("gated_qkv_store: unsupported dtype codes %d/%d", q_dt, c_dt);
#undef GQ_LAUNCH
    return 0;
}

// ============================================================== [q | k | v]: bias, norm per head, rotation, store
struct NormRotArgs {
    const float* proj; int ld;           // [T][ld] = [q: nh·d | k: nkv·d | v: nkv·vd | ...]; nkv 0: queries only
    const void* bias; int b_dt;          // over q, k, v; or null
    const void* qw; const void* kw; int w_dt;   // [d] weights of the heads' RMS norms, or null: no norm
    void* q_out; int q_dt;               // [T][nh·d]
    void* kpool; void* vpool; int c_dt;  // [pages][nkv][page_size][d], [pages][nkv][page_size][vd]
    const float* freq;                   // [rd/2] or null
    RowPlace pl;
    int T, nh, nkv, d, vd, rd, halves;   // halves: dim i pairs with dim i + rd/2, else dim 2i with dim 2i + 1
    float rot_mult, eps;
};

__device__ __forceinline__ float4 ld4_dt(const void* p, int dt, size_t i) {
    if (dt == SP_DT_F32) return *(const float4*)((const float*)p + i);
    const uint2 u = *(const uint2*)((const __nv_bfloat16*)p + i);
    const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&u.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&u.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, size_t i, float4 v) { *(float4*)(p + i) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, size_t i, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *(uint32_t*)&a; u.y = *(uint32_t*)&b;
    *(uint2*)(p + i) = u;
}

// One block per token, a warp per head in turn; a head's values wait in shared memory so that a lane reaches both dims of
// a pair. VEC: d, vd, rd/2 and all strides are multiples of four and pairs lie half apart: four neighbouring dims at a time.
constexpr int NR_WARPS = 8;
template <typename TO, typename TC, bool VEC>
__global__ void __launch_bounds__(NR_WARPS * 32) qkv_norm_rot_store_kernel(NormRotArgs a) {
    extern __shared__ __align__(16) float cs[];          // [2][rd/2], then [warps][d]
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int t = blockIdx.x;
    if (t >= a.T) return;
    const int pos = a.pl.positions[t];
    const int half = a.rd >> 1, d = a.d, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    pair_angles(cs, a.freq, half, pos, a.rot_mult);
    float* hv = cs + ((2 * half + 3) & ~3) + warp * ((d + 3) & ~3);
    __syncthreads();
    int page = 0;
    const bool place_ok = a.nkv > 0 && page_of(a.pl, t, pos, page);
    const int off = pos % a.pl.page_size;
    const float* src = a.proj + (size_t)t * a.ld;
    TO* q_out = (TO*)a.q_out + (size_t)t * a.nh * d;
    for (int h = warp; h < a.nh + a.nkv; h += NR_WARPS) {
        const bool is_q = h < a.nh;
        const void* w = is_q ? a.qw : a.kw;
        float ss = 0.0f;
        if (VEC) {
            for (int i = lane * 4; i < d; i += 128) {
                float4 v = *(const float4*)(src + h * d + i);
                if (a.bias) { const float4 b = ld4_dt(a.bias, a.b_dt, (size_t)h * d + i); v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w; }
                ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
                *(float4*)(hv + i) = v;
            }
        } else {
            for (int i = lane; i < d; i += 32) {
                const float v = src[h * d + i] + (a.bias ? sp_ld_dt(a.bias, a.b_dt, (size_t)h * d + i) : 0.0f);
                ss = fmaf(v, v, ss);
                hv[i] = v;
            }
        }
        if (w) {
            const float inv = 1.0f / sqrtf(sp_warp_sum(ss) / (float)d + a.eps);
            __syncwarp();
            for (int i = lane; i < d; i += 32) hv[i] = hv[i] * inv * sp_ld_dt(w, a.w_dt, i);
        }
        __syncwarp();
        const size_t base = is_q ? (size_t)h * d : (((size_t)page * a.nkv + (h - a.nh)) * a.pl.page_size + off) * d;
        if (VEC) {
            for (int i = lane * 4; i < d; i += 128) {
                float4 v = *(const float4*)(hv + i);
                if (i < a.rd) {
                    const bool lo = i < half;
                    const int p = lo ? i : i - half;
                    const float4 o = *(const float4*)(hv + (lo ? i + half : p)), c = *(const float4*)(cs + p);
                    float4 s4 = *(const float4*)(cs + half + p);
                    if (lo) { s4.x = -s4.x; s4.y = -s4.y; s4.z = -s4.z; s4.w = -s4.w; }
                    v.x = v.x * c.x + o.x * s4.x; v.y = v.y * c.y + o.y * s4.y; v.z = v.z * c.z + o.z * s4.z; v.w = v.w * c.w + o.w * s4.w;
                }
                if (is_q) st4(q_out, base + i, v);
                else if (place_ok) st4((TC*)a.kpool, base + i, v);
            }
        } else {
            for (int i = lane; i < d; i += 32) {
                float v = hv[i];
                if (i < a.rd) {
                    const bool lo = a.halves ? i < half : (i & 1) == 0;
                    const int p = a.halves ? (lo ? i : i - half) : i >> 1;
                    const int other = a.halves ? (lo ? i + half : p) : i ^ 1;
                    v = lo ? v * cs[p] - hv[other] * cs[half + p] : v * cs[p] + hv[other] * cs[half + p];
                }
                if (is_q) sp_st(q_out, base + i, v);
                else if (place_ok) sp_st((TC*)a.kpool, base + i, v);
            }
        }
        __syncwarp();
    }
    if (!place_ok) return;
    const int v0 = (a.nh + a.nkv) * d;
    for (int e = threadIdx.x * (VEC ? 4 : 1); e < a.nkv * a.vd; e += blockDim.x * (VEC ? 4 : 1)) {
        const int g = e / a.vd, r = e - g * a.vd;
        const size_t to = (((size_t)page * a.nkv + g) * a.pl.page_size + off) * a.vd + r;
        if (VEC) {
            float4 v = *(const float4*)(src + v0 + e);
            if (a.bias) { const float4 b = ld4_dt(a.bias, a.b_dt, (size_t)v0 + e); v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w; }
            st4((TC*)a.vpool, to, v);
        } else {
            sp_st((TC*)a.vpool, to, src[v0 + e] + (a.bias ? sp_ld_dt(a.bias, a.b_dt, (size_t)v0 + e) : 0.0f));
        }
    }
}

// The same where a head is one float4 per lane (d at most 128, pairs half apart, multiples of four): a warp asks for four
// heads' values at once, ahead of the angles, and a pair's other half comes from another lane.
template <typename TO, typename TC>
__global__ void __launch_bounds__(NR_WARPS * 32) qkv_norm_rot_rows_kernel(NormRotArgs a) {
    extern __shared__ __align__(16) float cs[];          // [2][rd/2]
    constexpr int HB = 4;
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int t = blockIdx.x;
    if (t >= a.T) return;
    const int half = a.rd >> 1, d = a.d, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int i = lane * 4, heads = a.nh + a.nkv;
    const bool in = i < d;
    const float* src = a.proj + (size_t)t * a.ld;
    const float4 z = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float4 v[HB];
    auto load = [&](int h0) {
#pragma unroll
        for (int u = 0; u < HB; ++u) {
            const int h = h0 + u * NR_WARPS;
            v[u] = (in && h < heads) ? *(const float4*)(src + h * d + i) : z;
        }
    };
    load(warp);
    const int pos = a.pl.positions[t];
    const float4 wq = a.qw && in ? ld4_dt(a.qw, a.w_dt, i) : z, wk = a.kw && in ? ld4_dt(a.kw, a.w_dt, i) : z;
    int page = 0;
    const bool place_ok = a.nkv > 0 && page_of(a.pl, t, pos, page);
    const int off = pos % a.pl.page_size;
    pair_angles(cs, a.freq, half, pos, a.rot_mult);
    __syncthreads();
    // the lane's four dims: their cos and sin, and the lane that holds their partners
    const bool turns = i < a.rd, lo = i < half;
    float4 c4 = make_float4(1.0f, 1.0f, 1.0f, 1.0f), s4 = z;
    if (turns) {
        c4 = *(const float4*)(cs + (lo ? i : i - half));
        s4 = *(const float4*)(cs + half + (lo ? i : i - half));
        if (lo) { s4.x = -s4.x; s4.y = -s4.y; s4.z = -s4.z; s4.w = -s4.w; }
    }
    const int peer = turns ? (lo ? lane + half / 4 : lane - half / 4) : lane;
    TO* q_out = (TO*)a.q_out + (size_t)t * a.nh * d;
    for (int h0 = warp; h0 < heads; h0 += HB * NR_WARPS) {
        if (h0 != warp) load(h0);
#pragma unroll
        for (int u = 0; u < HB; ++u) {
            const int h = h0 + u * NR_WARPS;
            if (h >= heads) break;
            const bool is_q = h < a.nh;
            if (a.bias && in) { const float4 b = ld4_dt(a.bias, a.b_dt, (size_t)h * d + i); v[u].x += b.x; v[u].y += b.y; v[u].z += b.z; v[u].w += b.w; }
            if (is_q ? a.qw != nullptr : a.kw != nullptr) {
                const float ss = sp_warp_sum((v[u].x * v[u].x + v[u].y * v[u].y) + (v[u].z * v[u].z + v[u].w * v[u].w));
                const float inv = 1.0f / sqrtf(ss / (float)d + a.eps);
                const float4 w = is_q ? wq : wk;
                v[u].x = v[u].x * inv * w.x; v[u].y = v[u].y * inv * w.y; v[u].z = v[u].z * inv * w.z; v[u].w = v[u].w * inv * w.w;
            }
            const float4 o = make_float4(__shfl_sync(0xffffffffu, v[u].x, peer), __shfl_sync(0xffffffffu, v[u].y, peer),
                                         __shfl_sync(0xffffffffu, v[u].z, peer), __shfl_sync(0xffffffffu, v[u].w, peer));
            if (!in) continue;
            if (turns) {
                v[u].x = v[u].x * c4.x + o.x * s4.x; v[u].y = v[u].y * c4.y + o.y * s4.y;
                v[u].z = v[u].z * c4.z + o.z * s4.z; v[u].w = v[u].w * c4.w + o.w * s4.w;
            }
            if (is_q) st4(q_out, (size_t)h * d + i, v[u]);
            else if (place_ok) st4((TC*)a.kpool, (((size_t)page * a.nkv + (h - a.nh)) * a.pl.page_size + off) * d + i, v[u]);
        }
    }
    if (!place_ok) return;
    const int v0 = heads * d;
    for (int e = threadIdx.x * 4; e < a.nkv * a.vd; e += blockDim.x * 4) {
        const int g = e / a.vd, r = e - g * a.vd;
        float4 x = *(const float4*)(src + v0 + e);
        if (a.bias) { const float4 b = ld4_dt(a.bias, a.b_dt, (size_t)v0 + e); x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w; }
        st4((TC*)a.vpool, (((size_t)page * a.nkv + g) * a.pl.page_size + off) * a.vd + r, x);
    }
}

SP_API int sp_qkv_norm_rot_store(const float* proj, int ld, const void* bias, int b_dt, const void* qw, const void* kw, int w_dt,
                                 void* q_out, int q_dt, void* kpool, void* vpool, int c_dt, const float* freq,
                                 const int* token_seq, const int* positions, const int* seq_row, const int* page_table,
                                 int max_pages, int page_size, int T, int nh, int nkv, int d, int vd, int rd, int halves,
                                 float rot_mult, float eps, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || vd <= 0 || rd < 0 || rd > d || (rd & 1)) SP_FAIL("qkv_norm_rot_store: the rotated dims %d must be even and at most %d", rd, d);
    if (rd > 0 && !freq) SP_FAIL("qkv_norm_rot_store: a frequency table is needed");
    if (ld < (nh + nkv) * d + nkv * vd) SP_FAIL("qkv_norm_rot_store: rows of %d numbers are too short", ld);
    NormRotArgs a{proj, ld, bias, b_dt, qw, kw, w_dt, q_out, q_dt, kpool, vpool, c_dt, freq,
                  RowPlace{token_seq, positions, seq_row, page_table, max_pages, page_size, sp_range_host},
                  T, nh, nkv, d, vd, rd, halves, rot_mult, eps};
    const bool vec = (halves || rd == 0) && d % 4 == 0 && vd % 4 == 0 && rd % 8 == 0 && ld % 4 == 0 &&
                     ((((uintptr_t)proj | (uintptr_t)bias | (uintptr_t)q_out | (uintptr_t)kpool | (uintptr_t)vpool) & 15) == 0);
    const size_t smem = (size_t)(((rd + 3) & ~3) + NR_WARPS * ((d + 3) & ~3)) * sizeof(float);
    if (smem > 48 * 1024) SP_FAIL("qkv_norm_rot_store: heads of %d are beyond this kernel's range", d);
#define NR_LAUNCH(TO, TC) do { if (vec && d <= 128) SP_CHECK_CALL("qkv_norm_rot_store", sp_launch_dependent(qkv_norm_rot_rows_kernel<TO, TC>, dim3(T), dim3(NR_WARPS * 32), (size_t)(rd > 0 ? rd : 4) * sizeof(float), stream, a)); \
    else if (vec) SP_CHECK_CALL("qkv_norm_rot_store", sp_launch_dependent(qkv_norm_rot_store_kernel<TO, TC, true>, dim3(T), dim3(NR_WARPS * 32), smem, stream, a)); \
    else SP_CHECK_CALL("qkv_norm_rot_store", sp_launch_dependent(qkv_norm_rot_store_kernel<TO, TC, false>, dim3(T), dim3(NR_WARPS * 32), smem, stream, a)); } while (0)
    if (q_dt == SP_DT_F32 && c_dt == SP_DT_F32) NR_LAUNCH(float, float);
    else if (q_dt == SP_DT_BF16 && c_dt == SP_DT_BF16) NR_LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else SP_FAIL("qkv_norm_rot_store: queries and cache share a storage type (codes %d/%d)", q_dt, c_dt);
#undef NR_LAUNCH
    return 0;
}

// ============================================================== [q | low-rank row | shared key part | gates]
struct LatentRotArgs {
    const float* proj; int ld;           // [T][ld] = [q: H·(d + rd) | row: rank | key part: rd | gates: H]; a reader has no row and no key part
    const void* wc; int w_dt;            // [rank] weight of the row's norm
    void* q_out; int q_dt;               // [T][H·(d + rd)], the rotated part of every head turned
    void* pool; int c_dt;                // [pages][page_size][rank + rd], or null (a reader)
    void* rows;                          // [T][rank + rd] like q_out, or null: the same rows token by token
    float* gates;                        // [T][H]
    const float* freq;                   // [rd/2]
    RowPlace pl;
    int T, H, d, rd, rank, halves;       // halves: dim i pairs with dim i + rd/2, else dim 2i with dim 2i + 1
    float rot_mult, eps;
};

__global__ void __launch_bounds__(256) latent_rot_store_kernel(LatentRotArgs a) {
    extern __shared__ float cs[];        // [2][rd/2]
    __shared__ float red[32];
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int t = blockIdx.x;
    if (t >= a.T) return;
    const int pos = a.pl.positions[t];
    const int half = a.rd >> 1;
    pair_angles(cs, a.freq, half, pos, a.rot_mult);
    __syncthreads();
    const float* src = a.proj + (size_t)t * a.ld;
    const int qd = a.d + a.rd, nq = a.H * qd;
    const int first = a.halves ? 1 : 2, apart = a.halves ? half : 1;      // pair i: dims first·i and first·i + apart
    // queries: the plain part passes, the rotated part turns pair by pair
    for (int e = threadIdx.x; e < a.H * a.d; e += blockDim.x) {
        const int h = e / a.d, i = e - h * a.d;
        sp_st_dt(a.q_out, a.q_dt, (size_t)t * nq + (size_t)h * qd + i, src[h * qd + i]);
    }
    for (int e = threadIdx.x; e < a.H * half; e += blockDim.x) {
        const int h = e / half, i = e - h * half;
        const int c = h * qd + a.d + first * i;
        const float u = src[c], v = src[c + apart], co = cs[i], si = cs[half + i];
        sp_st_dt(a.q_out, a.q_dt, (size_t)t * nq + c, u * co - v * si);
        sp_st_dt(a.q_out, a.q_dt, (size_t)t * nq + c + apart, v * co + u * si);
    }
    int g0 = nq;
    if (a.pool) {
        const float* lat = src + nq;
        float ss = 0.0f;
        for (int i = threadIdx.x; i < a.rank; i += blockDim.x) ss = fmaf(lat[i], lat[i], ss);
        ss = sp_block_sum(ss, red);
        const float inv = 1.0f / sqrtf(ss / (float)a.rank + a.eps);
        int page = 0;
        const bool place_ok = page_of(a.pl, t, pos, page);
        const int R = a.rank + a.rd;
        const size_t base = ((size_t)page * a.pl.page_size + pos % a.pl.page_size) * R;
        for (int i = threadIdx.x; i < a.rank; i += blockDim.x) {
            const float c = lat[i] * inv * sp_ld_dt(a.wc, a.w_dt, i);
            if (place_ok) sp_st_dt(a.pool, a.c_dt, base + i, c);
            if (a.rows) sp_st_dt(a.rows, a.q_dt, (size_t)t * R + i, c);
        }
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            const int c = a.rank + first * i;
            const float u = lat[c], v = lat[c + apart], co = cs[i], si = cs[half + i];
            const float ru = u * co - v * si, rv = v * co + u * si;
            if (place_ok) {
                sp_st_dt(a.pool, a.c_dt, base + c, ru);
                sp_st_dt(a.pool, a.c_dt, base + c + apart, rv);
            }
            if (a.rows) {
                sp_st_dt(a.rows, a.q_dt, (size_t)t * R + c, ru);
                sp_st_dt(a.rows, a.q_dt, (size_t)t * R + c + apart, rv);
            }
        }
        g0 += R;
    }
    if (a.gates)
        for (int h = threadIdx.x; h < a.H; h += blockDim.x) a.gates[(size_t)t * a.H + h] = src[g0 + h];
}

SP_API int sp_latent_rot_store(const float* proj, int ld, const void* wc, int w_dt, void* q_out, int q_dt, void* pool, int c_dt,
                               void* rows, float* gates, const float* freq, const int* token_seq, const int* positions,
                               const int* seq_row, const int* page_table, int max_pages, int page_size, int T, int H, int d,
                               int rd, int rank, int halves, float rot_mult, float eps, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || d <= 0 || rank <= 0 || rd < 0 || (rd & 1)) SP_FAIL("latent_rot_store: sizes %d heads x (%d + %d), rank %d", H, d, rd, rank);
    if (rd > 0 && !freq) SP_FAIL("latent_rot_store: a frequency table is needed");
    if (ld < H * (d + rd) + (pool ? rank + rd : 0) + (gates ? H : 0)) SP_FAIL("latent_rot_store: rows of %d numbers are too short", ld);
    if (pool && !wc) SP_FAIL("latent_rot_store: the row's norm needs its weight");
    LatentRotArgs a{proj, ld, wc, w_dt, q_out, q_dt, pool, c_dt, rows, gates, freq,
                    RowPlace{token_seq, positions, seq_row, page_table, max_pages, page_size, sp_range_host},
                    T, H, d, rd, rank, halves, rot_mult, eps};
    const size_t smem = (size_t)(rd > 0 ? rd : 2) * sizeof(float);
    SP_CHECK_CALL("latent_rot_store", sp_launch_dependent(latent_rot_store_kernel, dim3(T), dim3(256), smem, stream, a));
    return 0;
}

// ============================================================== gelu(z) times a gathered table row's part
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename TZ, typename TW>
__global__ void gelu_gather_mul_kernel(const TZ* __restrict__ z, const TW* __restrict__ table, const int* __restrict__ ids,
                                       TZ* __restrict__ out, int T, int C, int ld, int off, int vocab) {
    const size_t n = (size_t)T * C;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < n; e += (size_t)gridDim.x * blockDim.x) {
        const int t = (int)(e / C), j = (int)(e - (size_t)t * C);
        const int id = ids[t];
        const float s = (id >= 0 && id < vocab) ? sp_ld(table, (size_t)id * ld + off + j) : 0.0f;
        sp_st(out, e, gelu_tanh_f(sp_ld(z, e)) * s);
    }
}

SP_API int sp_gelu_gather_mul(const void* z, int z_dt, const void* table, int t_dt, const int* ids, void* out, int T, int C,
                              int ld, int off, int vocab, cudaStream_t stream) {
    if (T <= 0 || C <= 0) return 0;
    if (off < 0 || off + C > ld) SP_FAIL("gelu_gather_mul: columns %d..%d lie outside rows of %d", off, off + C, ld);
    const size_t n = (size_t)T * C;
    const int blocks = (int)((n + 255) / 256 > 148 * 16 ? 148 * 16 : (n + 255) / 256);
#define GG_LAUNCH(TZ, TW) gelu_gather_mul_kernel<TZ, TW><<<blocks, 256, 0, stream>>>((const TZ*)z, (const TW*)table, ids, (TZ*)out, T, C, ld, off, vocab)
    if (z_dt == SP_DT_F32 && t_dt == SP_DT_F32) GG_LAUNCH(float, float);
    else if (z_dt == SP_DT_BF16 && t_dt == SP_DT_BF16) GG_LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else if (z_dt == SP_DT_F32 && t_dt == SP_DT_BF16) GG_LAUNCH(float, __nv_bfloat16);
    else if (z_dt == SP_DT_BF16 && t_dt == SP_DT_F32) GG_LAUNCH(__nv_bfloat16, float);
    else SP_FAIL("gelu_gather_mul: unsupported dtype codes %d/%d", z_dt, t_dt);
#undef GG_LAUNCH
    SP_CHECK_LAUNCH("gelu_gather_mul");
    return 0;
}
