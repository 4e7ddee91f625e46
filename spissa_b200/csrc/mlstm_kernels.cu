// A matrix memory per head with exponential input gates and a running maximum (the mLSTM cell of xLSTM):
//
//   ĩ, f̃ = the token's two gate products plus bias;  i = c·tanh(ĩ / c),  f = log σ(c·tanh(f̃ / c))   (c = gate cap)
//   m_t = max(f + m_{t−1}, i),  m starts at 0;   S_t = e^{f + m_{t−1} − m_t} S_{t−1} + e^{i − m_t} k vᵀ;   n_t likewise with k
//   o = S_tᵀ q / (max(|n_t · q|, e^{−m_t}) + 1e-6)     q already times dim^(−1/2)
//   y = o / sqrt(mean(o²) + eps) ⊙ w ⊙ σ(g)             the mean over one head, w over all heads
//
// proj row (32-bit) = [q: H·d | k: H·d | v: H·vd | g: H·vd | ĩ: H | f̃: H]. State per slot, 32-bit: S [H][d][vd] and
// [H][d + 1] = (n, m). Everything but operands of the tensor-core form is 32-bit; the gates' running sums are 64-bit.
//
// Prompts run in chunks, all chunks in parallel. With F_i = Σ f and a_j = i_j − F_j counted from the chunk's start, m₀ the
// maximum in front of the chunk and M_i = max(m₀, max_{j ≤ i} a_j):  m_i = F_i + M_i, and
//     o_i  ~  e^{m₀ − M_i} q_i · S₀ + Σ_{j ≤ i} e^{a_j − M_i} (q_i · k_j) v_j
//     S_end = e^{m₀ − M_L} S₀ + Σ_j e^{a_j − M_L} k_j v_jᵀ
// so no running sum is left in any exponent but as a difference, and no exponent is positive. n is one more column of S
// (its "value" is 1), and n · q one more column of o.
#include "tcgen05.cuh"
#include "flash_common.cuh"

SP_API const char* sp_mlstm_last_error() { return sp_error_text; }
SP_DEFINE_RANGE_API(mlstm)

namespace {

struct MlArgs {
    const float* proj; int ld;
    const void* ib; const void* fb; const void* nw; int w_dt;   // [H], [H], [H·vd]
    float* S; float* nm; int n_slots;                            // [slots][H][d][vd], [slots][H][d + 1]
    void* out; int out_dt;                                       // [T][H·vd]
    const int* seq_start; const int* seq_slot;
    int B, T, H, d, vd, n_chunks;
    float cap, eps;
    // scratch of a prompt step
    float2* a2; float2* M2;         // [H][T] a_j and M_i as sums of two floats
    float* r; float* we; float* em; // [H][T] e^{m₀ − M_i}, e^{a_j − M_L}, e^{−m_i}
    float* ce;                      // [H][n_chunks] e^{m₀ − M_L}
    float* cs;                      // [n_chunks][H][d][vc] a chunk's own sum, then its start state; column vd is n
    float* raw;                     // [T][H][vc] outputs before the denominator; column vd is n · q
    int vc;                         // vd + 1 rounded up to a multiple of 4
    int* status;
};

__device__ __forceinline__ float ml_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_log_forget(float z, float cap) {
    const float c = cap * tanhf(z / cap);
    return fminf(c, 0.0f) - log1pf(expf(-fabsf(c)));
}

__device__ __forceinline__ bool ml_chunk_of(const MlArgs& a, int x, int ct, int& s, int& t0, int& n) {
    for (s = 0; s < a.B; ++s) {
        const int first = a.seq_start[s], cnt = a.seq_start[s + 1] - first;
        const int nc = (cnt + ct - 1) / ct;
        if (x < nc) {
            t0 = first + x * ct;
            n = min(ct, cnt - x * ct);
            return true;
        }
        x -= nc;
    }
    return false;
}

// ============================================================== the gates of a prompt step
// One block per (sequence, head); a warp takes 64 tokens, a lane two neighbouring ones, CT / 64 warps share a chunk; one warp
// carries the maximum from chunk to chunk (max-plus scan). Running sums and maxima in 64-bit; what the products read are
// exponentials of differences, each rounded once.
constexpr int MG_WARPS = 32;
template <int CT>
__global__ void __launch_bounds__(MG_WARPS * 32) mlstm_gates_kernel(MlArgs a) {
    static_assert(CT == 64 || CT == 128, "one or two warps of 64 tokens share a chunk");
    constexpr int WPC = CT / 64, CHUNKS = MG_WARPS / WPC;       // warps of a chunk, chunks of a pass
    __shared__ double sumF[MG_WARPS], topA[MG_WARPS], m0s[CHUNKS], m_run;
    sp_wait_for_predecessor();
    sp_allow_dependents();               // in this order: whoever starts from here on may read the projections at once
    const int s = blockIdx.x, h = blockIdx.y;
    const int slot = a.seq_slot[s];
    if (slot < 0 || slot >= a.n_slots) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, part = warp % WPC;
    const int first = a.seq_start[s], cnt = a.seq_start[s + 1] - first;
    int chunk0 = 0;
    for (int b = 0; b < s; ++b) chunk0 += (a.seq_start[b + 1] - a.seq_start[b] + CT - 1) / CT;
    const int nc = (cnt + CT - 1) / CT;
    float* m_state = a.nm + ((size_t)slot * a.H + h) * (a.d + 1) + a.d;
    if (threadIdx.x == 0) m_run = *m_state;
    const float ib = sp_ld_dt(a.ib, a.w_dt, h), fb = sp_ld_dt(a.fb, a.w_dt, h);
    const float* gates = a.proj + 2 * a.H * a.d + 2 * a.H * a.vd + h;
    for (int c0 = 0; c0 < nc; c0 += CHUNKS) {
        const int t = c0 * CT + warp * 64 + lane * 2;            // the lane's first token
        float iv[2], fv[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const float* row = gates + (size_t)(first + min(t + u, cnt - 1)) * a.ld;
            iv[u] = row[0];
            fv[u] = row[a.H];
        }
        double F[2], A[2], top[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            iv[u] = t + u < cnt ? ml_input_gate(iv[u] + ib, a.cap) : -INFINITY;
            fv[u] = t + u < cnt ? ml_log_forget(fv[u] + fb, a.cap) : 0.0f;
        }
        double inc = (double)fv[0] + (double)fv[1];              // inclusive over the lanes
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, inc, o);
            if (lane >= o) inc += up;
        }
        F[1] = inc;
        F[0] = inc - (double)fv[1];
        A[0] = (double)iv[0] - F[0];
        A[1] = (double)iv[1] - F[1];
        double mx = fmax(A[0], A[1]);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, mx, o);
            if (lane >= o) mx = fmax(mx, up);
        }
        double before = __shfl_up_sync(0xffffffffu, mx, 1);
        if (lane == 0) before = -INFINITY;
        top[0] = fmax(before, A[0]);
        top[1] = mx;
        if (lane == 31) { sumF[warp] = inc; topA[warp] = mx; }
        __syncthreads();
        if (warp == 0) {
            // chunk by chunk m ← max(m + S, T), S the chunk's sum of f, T = S + its largest a
            double S = 0.0, T = -INFINITY;
            if (lane < CHUNKS && c0 + lane < nc) {
#pragma unroll
                for (int w = 0; w < WPC; ++w) {
                    T = fmax(T, topA[lane * WPC + w] - S);
                    S += sumF[lane * WPC + w];
                }
                T += S;
            }
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double s1 = __shfl_up_sync(0xffffffffu, S, o), t1 = __shfl_up_sync(0xffffffffu, T, o);
                if (lane >= o) {
                    T = fmax(t1 + S, T);
                    S += s1;
                }
            }
            const double m_in = m_run, m_end = fmax(m_in + S, T);
            const double m_before = __shfl_up_sync(0xffffffffu, m_end, 1);
            if (lane < CHUNKS) m0s[lane] = lane == 0 ? m_in : m_before;
            if (lane == 31) m_run = m_end;                       // lanes beyond the last chunk add nothing
        }
        __syncthreads();
        const int c = c0 + warp / WPC;
        if (c < nc) {
            // of the chunk: the sum and the largest a in front of this warp's tokens, the largest of all
            const int w0 = warp - part;
            const double S = part ? sumF[w0] : 0.0, ahead = part ? topA[w0] : -INFINITY;
            const double all = WPC == 2 ? fmax(topA[w0], topA[w0 + WPC - 1] - sumF[w0]) : topA[w0];
            const double m0 = m0s[warp / WPC], ML = fmax(m0, all);
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                if (t + u >= cnt) break;
                const size_t at = (size_t)h * a.T + first + t + u;
                const double aj = A[u] - S, M = fmax(m0, fmax(ahead, top[u] - S));
                const float ah = (float)aj, mh = (float)M;
                a.a2[at] = make_float2(ah, (float)(aj - (double)ah));
                a.M2[at] = make_float2(mh, (float)(M - (double)mh));
                a.r[at] = expf((float)(m0 - M));
                a.we[at] = expf((float)(aj - ML));
                a.em[at] = expf((float)(-(F[u] + S + M)));
            }
            if (lane == 0 && part == 0) a.ce[(size_t)h * a.n_chunks + chunk0 + c] = expf((float)(m0 - ML));
        }
        __syncthreads();
    }
    if (threadIdx.x == 0) *m_state = (float)m_run;
}

// ============================================================== 32-bit products of a prompt step (any sizes)
constexpr int MC = 64;             // tokens of a chunk
constexpr int MP = 68;             // row stride of transposed tiles

// acc[u][v] += Σ_k a[k][4ty + u] · b[k][4tx + v]
__device__ __forceinline__ void ml_mm(const float* __restrict__ a, int lda, const float* __restrict__ b, int ldb, float (&acc)[4][4], int ty, int tx) {
    for (int k = 0; k < 64; ++k) {
        const float4 av = *(const float4*)(a + k * lda + 4 * ty), bv = *(const float4*)(b + k * ldb + 4 * tx);
        const float am[4] = {av.x, av.y, av.z, av.w}, bn[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int v = 0; v < 4; ++v) acc[u][v] = fmaf(am[u], bn[v], acc[u][v]);
    }
}

// a value row with its extra column: 1 at column vd
__device__ __forceinline__ float ml_value(const MlArgs& a, int t, int h, int col) {
    return col < a.vd ? a.proj[(size_t)t * a.ld + 2 * a.H * a.d + (size_t)h * a.vd + col] : (col == a.vd ? 1.0f : 0.0f);
}

// every chunk's own sum; grid (chunks, H, row blocks of 64 x column blocks of 64)
__global__ void __launch_bounds__(256) mlstm_sum_kernel(MlArgs a) {
    __shared__ __align__(16) float kd[MC][64], vv[MC][64];
    int s, t0, n;
    if (!ml_chunk_of(a, blockIdx.x, MC, s, t0, n)) return;
    const int h = blockIdx.y, nb = (a.vd + 64) / 64;
    const int e0 = (int)(blockIdx.z / nb) * 64, c0 = (int)(blockIdx.z % nb) * 64;
    for (int x = threadIdx.x; x < MC * 64; x += 256) {
        const int j = x >> 6, e = e0 + (x & 63), col = c0 + (x & 63);
        kd[j][x & 63] = (j < n && e < a.d) ? a.proj[(size_t)(t0 + j) * a.ld + (size_t)(a.H + h) * a.d + e] * a.we[(size_t)h * a.T + t0 + j] : 0.0f;
        vv[j][x & 63] = j < n ? ml_value(a, t0 + j, h, col) : 0.0f;
    }
    __syncthreads();
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[4][4] = {};
    ml_mm(&kd[0][0], 64, &vv[0][0], 64, acc, ty, tx);
    float* out = a.cs + ((size_t)blockIdx.x * a.H + h) * a.d * a.vc;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        const int e = e0 + 4 * ty + u;
        if (e >= a.d) continue;
#pragma unroll
        for (int v = 0; v < 4; ++v)
            if (c0 + 4 * tx + v < a.vc) out[(size_t)e * a.vc + c0 + 4 * tx + v] = acc[u][v];
    }
}

// the chunks' start states one after the other, element by element (the sums turn into start states in place); grid
// (sequences, H, blocks of 256 elements of [d][vc]). ``ct``: tokens of a chunk.
__global__ void __launch_bounds__(256) mlstm_scan_kernel(MlArgs a, int ct) {
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int s = blockIdx.x, h = blockIdx.y;
    const int x = blockIdx.z * 256 + threadIdx.x;
    if (x >= a.d * a.vc) return;
    const int slot = a.seq_slot[s];
    if (slot < 0 || slot >= a.n_slots) return;
    int first = 0;
    for (int b = 0; b < s; ++b) first += (a.seq_start[b + 1] - a.seq_start[b] + ct - 1) / ct;
    const int nc = (a.seq_start[s + 1] - a.seq_start[s] + ct - 1) / ct;
    const int e = x / a.vc, col = x - e * a.vc;
    if (col > a.vd) return;
    float* st = col < a.vd ? a.S + (((size_t)slot * a.H + h) * a.d + e) * a.vd + col
                           : a.nm + ((size_t)slot * a.H + h) * (a.d + 1) + e;
    float S = *st;
    const size_t step = (size_t)a.H * a.d * a.vc;
    float* cs = a.cs + (size_t)first * step + (size_t)h * a.d * a.vc + x;
    const float* ce = a.ce + (size_t)h * a.n_chunks + first;
    for (int k0 = 0; k0 < nc; k0 += 8) {
        float own[8], dv[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (k0 + u < nc) { own[u] = cs[(size_t)(k0 + u) * step]; dv[u] = ce[k0 + u]; }
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (k0 + u < nc) {
                cs[(size_t)(k0 + u) * step] = S;
                S = fmaf(dv[u], S, own[u]);
            }
    }
    *st = S;
}

// The same for the tensor-core form, four columns at a time (vd a multiple of four: the group that begins at column vd is n);
// the start states of the value columns leave as sums of two bfloat16 numbers, the high one in the lower half of a word, the
// low one above it. grid (sequences, H, blocks of 128 groups of [d][vc / 4])
__device__ __forceinline__ float pack_high_low(float v) {
    const __nv_bfloat16 hi = __float2bfloat16_rn(v);
    const __nv_bfloat162 both = __halves2bfloat162(hi, __float2bfloat16_rn(v - __bfloat162float(hi)));
    return __uint_as_float(*(const uint32_t*)&both);
}
__global__ void __launch_bounds__(128) mlstm_scan_packed_kernel(MlArgs a, int ct) {
    sp_wait_for_predecessor();
    sp_allow_dependents();               // whoever starts from here on may read the projections and the gates at once
    const int s = blockIdx.x, h = blockIdx.y, groups = a.vc / 4;
    const int x = blockIdx.z * 128 + threadIdx.x;
    if (x >= a.d * groups) return;
    const int slot = a.seq_slot[s];
    if (slot < 0 || slot >= a.n_slots) return;
    int first = 0;
    for (int b = 0; b < s; ++b) first += (a.seq_start[b + 1] - a.seq_start[b] + ct - 1) / ct;
    const int nc = (a.seq_start[s + 1] - a.seq_start[s] + ct - 1) / ct;
    const int e = x / groups, col = (x - e * groups) * 4;
    const bool value = col < a.vd;
    float* st = value ? a.S + (((size_t)slot * a.H + h) * a.d + e) * a.vd + col : a.nm + ((size_t)slot * a.H + h) * (a.d + 1) + e;
    float4 S = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (value) S = *(const float4*)st;
    else S.x = *st;
    const size_t step = (size_t)a.H * a.d * groups;
    float4* cs = (float4*)a.cs + (size_t)first * step + (size_t)h * a.d * groups + x;
    const float* ce = a.ce + (size_t)h * a.n_chunks + first;
    for (int k0 = 0; k0 < nc; k0 += 8) {
        float4 own[8];
        float dv[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (k0 + u < nc) { own[u] = cs[(size_t)(k0 + u) * step]; dv[u] = ce[k0 + u]; }
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (k0 + u < nc) {
                cs[(size_t)(k0 + u) * step] = value ? make_float4(pack_high_low(S.x), pack_high_low(S.y), pack_high_low(S.z), pack_high_low(S.w)) : S;
                S.x = fmaf(dv[u], S.x, own[u].x);
                S.y = fmaf(dv[u], S.y, own[u].y);
                S.z = fmaf(dv[u], S.z, own[u].z);
                S.w = fmaf(dv[u], S.w, own[u].w);
            }
    }
    if (value) *(float4*)st = S;
    else *st = S.x;
}

// outputs; grid (chunks, H, column blocks of 64)
__global__ void __launch_bounds__(256) mlstm_out_kernel(MlArgs a) {
    extern __shared__ __align__(16) float sm[];
    float* qT = sm;                     // [64][MP]   (dim, token), then P transposed (key, query)
    float* kT = qT + 64 * MP;           // [64][MP]
    float* Sb = kT + 64 * MP;           // [64][64]   start state, then values
    int s, t0, n;
    if (!ml_chunk_of(a, blockIdx.x, MC, s, t0, n)) return;
    const int h = blockIdx.y, c0 = blockIdx.z * 64;
    const float qscale = 1.0f / sqrtf((float)a.d);
    const float* cs = a.cs + ((size_t)blockIdx.x * a.H + h) * a.d * a.vc;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float p[4][4] = {}, acc[4][4] = {};
    for (int e0 = 0; e0 < a.d; e0 += 64) {
        __syncthreads();
        for (int x = threadIdx.x; x < MC * 64; x += 256) {
            const int i = x >> 6, e = e0 + (x & 63);
            const bool in = i < n && e < a.d;
            const float* row = a.proj + (size_t)(t0 + (in ? i : 0)) * a.ld + (size_t)h * a.d + e;
            qT[(x & 63) * MP + i] = in ? row[0] * qscale : 0.0f;
            kT[(x & 63) * MP + i] = in ? row[(size_t)a.H * a.d] : 0.0f;
            const int se = e0 + (x >> 6), col = c0 + (x & 63);
            Sb[x] = (se < a.d && col <= a.vd) ? cs[(size_t)se * a.vc + col] : 0.0f;
        }
        __syncthreads();
        ml_mm(qT, MP, kT, MP, p, ty, tx);
        ml_mm(qT, MP, Sb, 64, acc, ty, tx);
    }
    __syncthreads();
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        const int i = 4 * ty + u;
        const size_t at = (size_t)h * a.T + t0 + min(i, n - 1);
        const float2 M = a.M2[at];
        const float r = a.r[at];
#pragma unroll
        for (int v = 0; v < 4; ++v) {
            const int j = 4 * tx + v;
            float w = 0.0f;
            if (j <= i && i < n) {
                const float2 aj = a.a2[(size_t)h * a.T + t0 + j];
                w = p[u][v] * expf((aj.x - M.x) + (aj.y - M.y));
            }
            qT[j * MP + i] = w;
            acc[u][v] *= r;
        }
    }
    for (int x = threadIdx.x; x < MC * 64; x += 256) Sb[x] = (x >> 6) < n ? ml_value(a, t0 + (x >> 6), h, c0 + (x & 63)) : 0.0f;
    __syncthreads();
    ml_mm(qT, MP, Sb, 64, acc, ty, tx);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        const int i = 4 * ty + u;
        if (i >= n) continue;
#pragma unroll
        for (int v = 0; v < 4; ++v)
            if (c0 + 4 * tx + v <= a.vd) a.raw[((size_t)(t0 + i) * a.H + h) * a.vc + c0 + 4 * tx + v] = acc[u][v];
    }
}

// denominator, unit rms, weight, gate, store; grid (T, H)
__global__ void __launch_bounds__(128) mlstm_finish_kernel(MlArgs a) {
    __shared__ float red[32];
    const int t = blockIdx.x, h = blockIdx.y;
    const float* o = a.raw + ((size_t)t * a.H + h) * a.vc;
    const float inv_den = 1.0f / (fmaxf(fabsf(o[a.vd]), a.em[(size_t)h * a.T + t]) + 1e-6f);
    float ss = 0.0f;
    for (int c = threadIdx.x; c < a.vd; c += blockDim.x) {
        const float v = o[c] * inv_den;
        ss = fmaf(v, v, ss);
    }
    ss = sp_block_sum(ss, red);
    const float f = inv_den / sqrtf(ss / (float)a.vd + a.eps);
    const float* g = a.proj + (size_t)t * a.ld + 2 * a.H * a.d + (size_t)(a.H + h) * a.vd;
    for (int c = threadIdx.x; c < a.vd; c += blockDim.x)
        sp_st_dt(a.out, a.out_dt, ((size_t)t * a.H + h) * a.vd + c, o[c] * f * sp_ld_dt(a.nw, a.w_dt, (size_t)h * a.vd + c) / (1.0f + expf(-g[c])));
}

// ============================================================== the products of a prompt step on tcgen05
// Chunks of 128 tokens; q, k and v as bfloat16 (projections), everything that carries a gate or a state as the sum of two
// bfloat16 numbers, 32-bit accumulators in tensor memory. Operands are written into shared memory by the threads in the
// 128-byte swizzle (rows of 64 numbers, 16-byte pieces exchanged by the row's low bits).
constexpr int TK = 128;
constexpr int BOX = TK * 128;                 // bytes of 128 rows of 64 numbers
constexpr int OT_LD = 260;                    // floats of a row of results in shared memory (rows 16 bytes apart in the banks)

__device__ __forceinline__ uint32_t sw_at(int row, int piece) { return (uint32_t)(row * 128 + ((piece ^ (row & 7)) << 4)); }
__device__ __forceinline__ uint4 pack8(const float (&f)[8]) {
    return make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}
__device__ __forceinline__ void low_parts(float (&f)[8], const uint4& hi) {
    const uint32_t w[4] = {hi.x, hi.y, hi.z, hi.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        f[2 * i] -= __uint_as_float(w[i] << 16);
        f[2 * i + 1] -= __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void load8(const float* p, bool in, float (&f)[8]) {
    const float4 z = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    const float4 a = in ? *(const float4*)p : z, b = in ? *(const float4*)(p + 4) : z;
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void proxy_fence() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

// A chunk's values, columns c0 .. c0 + nb - 1 of head h, as boxes of 64 columns with one row per token (the product's K):
// 4,096 pieces of eight numbers over the THREADS of a block, a thread's pieces u0 .. u0 + N - 1. All of a batch's loads come before its stores,
// which the compiler would not let them pass.
template <int N, int THREADS = 256>
__device__ __forceinline__ void load_values(const MlArgs& a, float4 (&r)[2 * N], int u0, int h, int t0, int n, int c0, int nb) {
#pragma unroll
    for (int u = 0; u < N; ++u) {
        const int x = threadIdx.x + THREADS * (u0 + u), j = x >> 5, col = c0 + 8 * (x & 31);
        const float4* p = (const float4*)(a.proj + (size_t)(t0 + j) * a.ld + 2 * a.H * a.d + (size_t)h * a.vd + col);
        const bool in = j < n && col < a.vd;
        r[2 * u] = in ? p[0] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        r[2 * u + 1] = in ? p[1] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
}
__device__ __forceinline__ uint4 pack8(const float4& a, const float4& b) {
    return make_uint4(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w), pack_bf16(b.x, b.y), pack_bf16(b.z, b.w));
}
template <int N, int THREADS = 256>
__device__ __forceinline__ void store_values(uint8_t* dst, const float4 (&r)[2 * N], int u0, int nb) {
#pragma unroll
    for (int u = 0; u < N; ++u) {
        const int x = threadIdx.x + THREADS * (u0 + u), j = x >> 5, c = x & 31;
        if (8 * c < nb) *(uint4*)(dst + (c >> 3) * BOX + sw_at(j, c & 7)) = pack8(r[2 * u], r[2 * u + 1]);
    }
}

// every chunk's own sum: [128 key dims] x [up to 256 value columns] over the chunk's tokens, keys times e^{a_j − M_L} as high
// and low parts, both operands with the tokens as rows. n (the sum of the weighted keys) is added up in 32-bit on the way.
// grid (chunks, H, row blocks of 128 x column blocks of 256)
__global__ void __launch_bounds__(256) mlstm_sum_tc_kernel(MlArgs a) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t bar;
    __shared__ uint32_t tmem_slot;
    __shared__ int gave_up;
    __shared__ float part[16][TK + 1];
    uint8_t* sm = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    uint8_t *kh = sm, *kl = sm + 2 * BOX, *vs = sm + 4 * BOX;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        gave_up = 0;
        mbar_init(smem_u32(&bar), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        proxy_fence();
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(256u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    sp_allow_dependents();
    int s, t0 = 0, n = 0;
    const bool live = ml_chunk_of(a, blockIdx.x, TK, s, t0, n);
    const int h = blockIdx.y, cb = (a.vd + 255) / 256;
    const int e0 = (int)(blockIdx.z / cb) * TK, c0 = (int)(blockIdx.z % cb) * 256;
    const int nb = (min(256, a.vd - c0) + 15) / 16 * 16;
    float* out = a.cs + ((size_t)blockIdx.x * a.H + h) * a.d * a.vc;
    if (live) {
        // keys and values come from the projections, which are complete when this kernel starts; the gates are waited for
        const int c8 = threadIdx.x & 15, tg = threadIdx.x >> 4, e = e0 + 8 * c8;
        float4 kr[16], vr[16];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int j = tg + 16 * u;
            const bool in = j < n && e < a.d;
            const float4* p = (const float4*)(a.proj + (size_t)(t0 + j) * a.ld + (size_t)(a.H + h) * a.d + e);
            kr[2 * u] = in ? p[0] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            kr[2 * u + 1] = in ? p[1] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        load_values<8>(a, vr, 0, h, t0, n, c0, nb);
        store_values<8>(vs, vr, 0, nb);
        load_values<8>(a, vr, 8, h, t0, n, c0, nb);
        sp_wait_for_predecessor();
        float ns[8] = {}, w[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) w[u] = tg + 16 * u < n ? a.we[(size_t)h * a.T + t0 + tg + 16 * u] : 0.0f;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            float f[8] = {kr[2 * u].x, kr[2 * u].y, kr[2 * u].z, kr[2 * u].w, kr[2 * u + 1].x, kr[2 * u + 1].y, kr[2 * u + 1].z, kr[2 * u + 1].w};
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                f[i] *= w[u];
                ns[i] += f[i];
            }
            const uint4 hi = pack8(f);
            low_parts(f, hi);
            const uint32_t at = (uint32_t)((c8 >> 3) * BOX) + sw_at(tg + 16 * u, c8 & 7);
            *(uint4*)(kh + at) = hi;
            *(uint4*)(kl + at) = pack8(f);
        }
        store_values<8>(vs, vr, 8, nb);
#pragma unroll
        for (int i = 0; i < 8; ++i) part[tg][8 * c8 + i] = ns[i];
        proxy_fence();
    }
    __syncthreads();
    if (live && threadIdx.x == 0) {
        const uint32_t idesc = umma_idesc_bf16_bmn(TK, nb) | (1u << 15);        // both operands with K (the tokens) as rows
        const int ks = (n + 15) / 16;
        for (int lo = 0; lo < 2; ++lo)
            for (int k = 0; k < ks; ++k)
                tc_mma_bf16(tmem, umma_desc_mn_sw128(smem_u32(lo ? kl : kh) + k * 2048, BOX), umma_desc_mn_sw128(smem_u32(vs) + k * 2048, BOX), idesc,
                            (lo | k) ? 1u : 0u);
        tc_commit(smem_u32(&bar));
    }
    if (live) {
        if (c0 == 0 && threadIdx.x < TK && e0 + (int)threadIdx.x < a.d) {
            float sum = 0.0f;
#pragma unroll
            for (int g = 0; g < 16; ++g) sum += part[g][threadIdx.x];
            out[(size_t)(e0 + threadIdx.x) * a.vc + a.vd] = sum;
        }
        const bool ok = mbar_wait_flag(smem_u32(&bar), 0, a.status, 151, &gave_up);
        tc_fence_after();
        // through shared memory (the products have read theirs), so that the sums leave as whole lines
        float* rows = (float*)sm;
        for (int c = (warp >> 2) * 32; c < nb; c += 64) {
            uint32_t r[32];
            tc_ld_32x32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + c, r);
            tc_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; i += 4)
                *(float4*)(rows + ((warp & 3) * 32 + lane) * OT_LD + c + i) =
                    make_float4(__uint_as_float(r[i]), __uint_as_float(r[i + 1]), __uint_as_float(r[i + 2]), __uint_as_float(r[i + 3]));
        }
        __syncthreads();
        if (ok) {
#pragma unroll 4
            for (int x = threadIdx.x; x < TK * 64; x += 256) {
                const int e = x >> 6, c = (x & 63) * 4;
                if (e0 + e < a.d && c0 + c < a.vd && c < nb) *(float4*)(out + (size_t)(e0 + e) * a.vc + c0 + c) = *(const float4*)(rows + e * OT_LD + c);
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(256u) : "memory");
    }
}

// Outputs of a chunk, up to 256 value columns. Blocks of 64 key dims pass through two shared-memory stages (q, k, the start
// state's high and low part): A = q kᵀ and O = q · S₀ gather in tensor memory; the rows of O take e^{m₀ − M_i}, A turns into
// the pair weights (high and low part, as an operand in tensor memory), the values follow into the stage that is free, and O
// gathers the chunk's own share. A thread owns a row (token) and every fourth group of 32 columns; warps whose
// numbers are equal modulo 4 share rows. With one column block the denominator, the unit rms, weight and gate follow here, else the raw outputs leave.
// grid (chunks, H, column blocks of 256)
constexpr int OT_THREADS = 512;
constexpr int OT_STAGE = 2 * BOX + 2 * 32768;
static_assert(TK * OT_LD * 4 <= 2 * OT_STAGE, "the outputs reuse the operands' stages");
__global__ void __launch_bounds__(OT_THREADS) mlstm_out_tc_kernel(MlArgs a) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t bar_free[2], bar_a, bar_o;
    __shared__ uint32_t tmem_slot;
    __shared__ int gave_up;
    __shared__ float2 aj[TK];
    __shared__ float nvec[2][64], qn_s[4][TK], ss_s[4][TK];
    uint8_t* sm = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        gave_up = 0;
        mbar_init(smem_u32(&bar_free[0]), 1);
        mbar_init(smem_u32(&bar_free[1]), 1);
        mbar_init(smem_u32(&bar_a), 1);
        mbar_init(smem_u32(&bar_o), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        proxy_fence();
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    constexpr uint32_t COL_A = 0, COL_PH = 128, COL_PL = 192, COL_O = 256;
    sp_allow_dependents();
    int s, t0 = 0, n = 0;
    const bool live = ml_chunk_of(a, blockIdx.x, TK, s, t0, n);
    if (live) {
        const int h = blockIdx.y, c0 = blockIdx.z * 256, d = a.d;
        const int nv = min(256, a.vd - c0), nb = (nv + 15) / 16 * 16;
        const int row = (warp & 3) * 32 + lane, hh = warp >> 2;
        const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
        const float qscale = 1.0f / sqrtf((float)d);
        const bool mine = row < n;
        const float* cs = a.cs + ((size_t)blockIdx.x * a.H + h) * d * a.vc;
        const uint32_t id_a = umma_idesc_bf16(TK, TK), id_o = umma_idesc_bf16_bmn(TK, nb);
        const int nE = (d + 63) / 64;
        bool ok = true;
        float dot = 0.0f;
        // 256 bytes of operands per thread: q, k and the start state of a block of key dims, in the end the values; the next
        // ones are asked for before the products of the ones at hand begin
        float4 buf[16];
        const float4 z4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        auto load_qk = [&](int eb) {
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int x = threadIdx.x + OT_THREADS * u, j = x >> 3, e = eb * 64 + 8 * (x & 7);
                const bool in = j < n && e < d;
                const float4 *pq = (const float4*)(a.proj + (size_t)(t0 + j) * a.ld + (size_t)h * d + e), *pk = (const float4*)((const float*)pq + (size_t)a.H * d);
                buf[4 * u] = in ? pq[0] : z4;
                buf[4 * u + 1] = in ? pq[1] : z4;
                buf[4 * u + 2] = in ? pk[0] : z4;
                buf[4 * u + 3] = in ? pk[1] : z4;
            }
        };
        auto load_state = [&](int eb) {
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int x = threadIdx.x + OT_THREADS * u, e = eb * 64 + (x >> 5), col = c0 + 8 * (x & 31);
                const bool in = e < d && col < a.vd;
                const float4* p = (const float4*)(cs + (size_t)e * a.vc + col);
                buf[8 + 2 * u] = in ? p[0] : z4;
                buf[9 + 2 * u] = in ? p[1] : z4;
            }
        };
        auto store_qk = [&](uint8_t* q, uint8_t* k) {
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int x = threadIdx.x + OT_THREADS * u;
                *(uint4*)(q + sw_at(x >> 3, x & 7)) = pack8(buf[4 * u], buf[4 * u + 1]);
                *(uint4*)(k + sw_at(x >> 3, x & 7)) = pack8(buf[4 * u + 2], buf[4 * u + 3]);
            }
        };
        auto store_state = [&](uint8_t* sh, uint8_t* sl) {
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int x = threadIdx.x + OT_THREADS * u, r = x >> 5, c = x & 31;
                if (8 * c >= nb) continue;
                const uint4 w0 = *(const uint4*)&buf[8 + 2 * u], w1 = *(const uint4*)&buf[9 + 2 * u];
                const uint32_t to = (uint32_t)((c >> 3) * 8192) + sw_at(r, c & 7);
                *(uint4*)(sh + to) = make_uint4(__byte_perm(w0.x, w0.y, 0x5410), __byte_perm(w0.z, w0.w, 0x5410), __byte_perm(w1.x, w1.y, 0x5410), __byte_perm(w1.z, w1.w, 0x5410));
                *(uint4*)(sl + to) = make_uint4(__byte_perm(w0.x, w0.y, 0x7632), __byte_perm(w0.z, w0.w, 0x7632), __byte_perm(w1.x, w1.y, 0x7632), __byte_perm(w1.z, w1.w, 0x7632));
            }
        };
        // the projections and the gates are complete when this kernel starts; the start states are waited for
        load_qk(0);
        const size_t at = (size_t)h * a.T + t0 + (mine ? row : 0);
        const float2 M = a.M2[at];
        const float rq = a.r[at] * qscale, em = a.em[at];
        if (threadIdx.x < TK) aj[threadIdx.x] = (int)threadIdx.x < n ? a.a2[(size_t)h * a.T + t0 + threadIdx.x] : make_float2(0.0f, 0.0f);
        sp_wait_for_predecessor();
        load_state(0);
        for (int eb = 0; eb < nE; ++eb) {
            uint8_t *q = sm + (eb & 1) * OT_STAGE, *k = q + BOX, *sh = q + 2 * BOX, *sl = sh + 32768;
            if (eb >= 2) ok = mbar_wait_flag(smem_u32(&bar_free[eb & 1]), (uint32_t)((eb >> 1) - 1) & 1u, a.status, 152, &gave_up) && ok;
            if (threadIdx.x < 64) nvec[eb & 1][threadIdx.x] = eb * 64 + (int)threadIdx.x < d ? cs[(size_t)(eb * 64 + threadIdx.x) * a.vc + a.vd] : 0.0f;
            store_qk(q, k);
            store_state(sh, sl);
            if (eb + 1 < nE) {
                load_qk(eb + 1);
                load_state(eb + 1);
            } else {
                load_values<8, OT_THREADS>(a, buf, 0, h, t0, n, c0, nb);
            }
            proxy_fence();
            __syncthreads();
            if (threadIdx.x == 0) {
                const int ks = min(4, (d - eb * 64 + 15) / 16);
                for (int i = 0; i < ks; ++i) {
                    const uint64_t dq = umma_desc_sw128(smem_u32(q)) + 2 * i;
                    tc_mma_bf16(tmem + COL_A, dq, umma_desc_sw128(smem_u32(k)) + 2 * i, id_a, (eb | i) ? 1u : 0u);
                    tc_mma_bf16(tmem + COL_O, dq, umma_desc_mn_sw128(smem_u32(sh) + i * 2048, 8192), id_o, (eb | i) ? 1u : 0u);
                    tc_mma_bf16(tmem + COL_O, dq, umma_desc_mn_sw128(smem_u32(sl) + i * 2048, 8192), id_o, 1u);
                }
                tc_commit(smem_u32(&bar_free[eb & 1]));
                if (eb == nE - 1) tc_commit(smem_u32(&bar_a));
            }
            // q · n of the row, a quarter of the block's dims each
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const uint4 w = *(const uint4*)(q + sw_at(row, hh * 2 + c));
                const uint32_t v[4] = {w.x, w.y, w.z, w.w};
                const float* nr = &nvec[eb & 1][hh * 16 + c * 8];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    dot = fmaf(__uint_as_float(v[i] << 16), nr[2 * i], dot);
                    dot = fmaf(__uint_as_float(v[i] & 0xffff0000u), nr[2 * i + 1], dot);
                }
            }
        }
        // the values go where block nE - 2 was
        uint8_t* vs = sm + (nE & 1) * OT_STAGE;
        if (nE >= 2) ok = mbar_wait_flag(smem_u32(&bar_free[nE & 1]), (uint32_t)((nE - 2) >> 1) & 1u, a.status, 152, &gave_up) && ok;
        store_values<8, OT_THREADS>(vs, buf, 0, nb);
        proxy_fence();
        ok = mbar_wait_flag(smem_u32(&bar_a), 0, a.status, 153, &gave_up) && ok;
        tc_fence_after();
        float qn = dot * rq;
        {
            uint32_t x[32], ph[16], pl[16];
            tc_ld_32x32(tmem + lanes + COL_A + hh * 32, x);
            tc_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
                float w[2];
#pragma unroll
                for (int v = 0; v < 2; ++v) {
                    const int j = hh * 32 + i + v;
                    const float2 e = aj[j];
                    w[v] = (mine && j <= row) ? __uint_as_float(x[i + v]) * qscale * __expf((e.x - M.x) + (e.y - M.y)) : 0.0f;
                    qn += w[v];
                }
                const uint32_t hi = pack_bf16(w[0], w[1]);
                ph[i >> 1] = hi;
                pl[i >> 1] = pack_bf16(w[0] - __uint_as_float(hi << 16), w[1] - __uint_as_float(hi & 0xffff0000u));
            }
            tc_st_32x16(tmem + lanes + COL_PH + hh * 16, ph);
            tc_st_32x16(tmem + lanes + COL_PL + hh * 16, pl);
        }
#pragma unroll 1
        for (int c = hh * 32; c < nb; c += 128) {
            uint32_t x[32];
            tc_ld_32x32(tmem + lanes + COL_O + c, x);
            tc_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) x[i] = __float_as_uint(__uint_as_float(x[i]) * rq);
            tc_st_32x32(tmem + lanes + COL_O + c, x);
        }
        tc_st_wait();
        qn_s[hh][row] = qn;
        tc_fence_before();
        __syncthreads();
        if (threadIdx.x == 0) {
            tc_fence_after();
            const int ks = (n + 15) / 16;
            for (int lo = 0; lo < 2; ++lo)
                for (int k = 0; k < ks; ++k)
                    tc_mma_bf16_ts(tmem + COL_O, tmem + (lo ? COL_PL : COL_PH) + 8 * k, umma_desc_mn_sw128(smem_u32(vs) + k * 2048, BOX), id_o, 1u);
            tc_commit(smem_u32(&bar_o));
        }
        qn = (qn_s[0][row] + qn_s[1][row]) + (qn_s[2][row] + qn_s[3][row]);
        const bool whole = gridDim.z == 1;
        const float inv_den = 1.0f / (fmaxf(fabsf(qn), em) + 1e-6f);
        ok = mbar_wait_flag(smem_u32(&bar_o), 0, a.status, 154, &gave_up) && ok;
        tc_fence_after();
        float f = 1.0f;
        if (whole) {
            float ss = 0.0f;
#pragma unroll 1
            for (int c = hh * 32; c < nb; c += 128) {
                uint32_t x[32];
                tc_ld_32x32(tmem + lanes + COL_O + c, x);
                tc_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    const float o = __uint_as_float(x[i]) * inv_den;
                    if (c + i < nv) ss = fmaf(o, o, ss);
                }
            }
            ss_s[hh][row] = ss;
            __syncthreads();
            f = inv_den / sqrtf(((ss_s[0][row] + ss_s[1][row]) + (ss_s[2][row] + ss_s[3][row])) / (float)a.vd + a.eps);
        }
        float* raw = a.raw + ((size_t)(t0 + row) * a.H + h) * a.vc;
        if (!whole && ok && mine && c0 == 0 && hh == 0) raw[a.vd] = qn;
        // the rows pass through shared memory (all products have read theirs), so that gates and outputs move as whole lines
        float* rows = (float*)sm;
#pragma unroll 1
        for (int c = hh * 32; c < nb; c += 128) {
            uint32_t x[32];
            tc_ld_32x32(tmem + lanes + COL_O + c, x);
            tc_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; i += 4)
                *(float4*)(rows + row * OT_LD + c + i) = make_float4(__uint_as_float(x[i]) * f, __uint_as_float(x[i + 1]) * f,
                                                                     __uint_as_float(x[i + 2]) * f, __uint_as_float(x[i + 3]) * f);
        }
        __syncthreads();
        const int col = lane * 8;
        if (ok && col < nv) {
            float wv[8];
            load8((const float*)a.nw + (size_t)h * a.vd + c0 + col, true, wv);
#pragma unroll 4
            for (int u = 0; u < TK / 16; ++u) {
                const int j = warp + 16 * u;
                if (j >= n) break;
                const size_t to = (size_t)(t0 + j) * a.H + h;
                float y[8];
                load8(rows + j * OT_LD + col, true, y);
                if (!whole) {
                    *(float4*)(a.raw + to * a.vc + c0 + col) = make_float4(y[0], y[1], y[2], y[3]);
                    *(float4*)(a.raw + to * a.vc + c0 + col + 4) = make_float4(y[4], y[5], y[6], y[7]);
                    continue;
                }
                float gv[8];
                load8(a.proj + (size_t)(t0 + j) * a.ld + 2 * a.H * d + (size_t)(a.H + h) * a.vd + col, true, gv);
#pragma unroll
                for (int v = 0; v < 8; ++v) y[v] = __fdividef(y[v] * wv[v], 1.0f + __expf(-gv[v]));
                *(uint4*)((__nv_bfloat16*)a.out + to * a.vd + col) = pack8(y);
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

// ============================================================== one token per sequence
// A cluster of CTAs per (head, sequence) shares the value columns out; each streams its columns of S once (on their way
// into L2 before the projections are there), all compute n · q, the first one writes n
// and m once everybody has read them, and every CTA sends the squares of its outputs to all others' shared memory.
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ void store_peer_f32(float* p, uint32_t rank, float v) {
    uint32_t remote;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(smem_u32(p)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(v) : "memory");
}

constexpr int MS_COLS = 32;        // value columns of a CTA and pass
// VEC: neighbouring columns of a thread (4: 16-byte accesses); threads are (32 / VEC) columns x ROWS rows
template <int VEC>
__global__ void __launch_bounds__(256) mlstm_step_kernel(MlArgs a, int cz) {
    constexpr int XT = MS_COLS / VEC, ROWS = 256 / XT, AHEAD = 4;
    constexpr int PARTS = VEC == 4 ? 8 : ROWS;            // partial sums of a column that meet in shared memory
    extern __shared__ __align__(16) float sm[];
    float* qs = sm;                      // [d]
    float* ks = qs + ((a.d + 3) & ~3);   // [d]
    float* red = ks + ((a.d + 3) & ~3);  // [PARTS][32]
    float* oc = red + PARTS * MS_COLS;   // [column passes][32] this CTA's outputs
    __shared__ float scratch[32], ssq[8];
    const int rank = blockIdx.x, h = blockIdx.y, s = blockIdx.z;
    const int x = threadIdx.x % XT, y = threadIdx.x / XT;
    const int d = a.d, vd = a.vd, Hd = a.H * d, Hv = a.H * vd;
    const int slot = a.seq_slot[s];
    const bool live = slot >= 0 && slot < a.n_slots;          // the same for a whole cluster
    float* gS = a.S + ((size_t)(live ? slot : 0) * a.H + h) * d * vd;
    float* gn = a.nm + ((size_t)(live ? slot : 0) * a.H + h) * (d + 1);
    const int passes = (vd + MS_COLS * cz - 1) / (MS_COLS * cz);
    float st[AHEAD][VEC];
    auto load = [&](int col, int e0) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int e = e0 + u * ROWS;
            if (VEC == 4) {
                const float4 f = (e < d && col < vd) ? *(const float4*)(gS + (size_t)e * vd + col) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                st[u][0] = f.x; st[u][VEC > 1 ? 1 : 0] = f.y; st[u][VEC > 2 ? 2 : 0] = f.z; st[u][VEC > 3 ? 3 : 0] = f.w;
            } else {
                st[u][0] = (e < d && col < vd) ? gS[(size_t)e * vd + col] : 0.0f;
            }
        }
    };
    sp_allow_dependents();
    if (cz > 1) cluster_arrive();                         // everybody has started: waited for before anything is sent
    for (int e = threadIdx.x; e < d; e += 256)            // the first pass's columns on their way into L2
        if (rank * MS_COLS < vd) asm volatile("prefetch.global.L2 [%0];" ::"l"(gS + (size_t)e * vd + rank * MS_COLS));
    sp_wait_for_predecessor();
    load(rank * MS_COLS + x * VEC, y);
    const int t = a.seq_start[s];
    const float* row = a.proj + (size_t)t * a.ld;
    const float ig = ml_input_gate(row[2 * Hd + 2 * Hv + h] + sp_ld_dt(a.ib, a.w_dt, h), a.cap);
    const float fg = ml_log_forget(row[2 * Hd + 2 * Hv + a.H + h] + sp_ld_dt(a.fb, a.w_dt, h), a.cap);
    const float m0 = gn[d];
    const float m1 = fmaxf(fg + m0, ig);
    const float keep = expf(fg + m0 - m1), take = expf(ig - m1);
    const float qscale = 1.0f / sqrtf((float)d);
    float nq = 0.0f;
    for (int e = threadIdx.x; e < d; e += 256) {
        const float q = row[h * d + e] * qscale, k = row[Hd + h * d + e];
        qs[e] = q;
        ks[e] = take * k;
        nq = fmaf(fmaf(keep, gn[e], take * k), q, nq);
    }
    // the output's gate and weight of the first pass, asked for ahead of their use
    const float* g = row + 2 * Hd + Hv + (size_t)h * vd;
    const int own = rank * MS_COLS + threadIdx.x;
    float gate = 0.0f, weight = 0.0f;
    if (threadIdx.x < MS_COLS && own < vd) {
        gate = g[own];
        weight = sp_ld_dt(a.nw, a.w_dt, (size_t)h * vd + own);
    }
    nq = sp_block_sum(nq, scratch);
    const float inv_den = 1.0f / (fmaxf(fabsf(nq), expf(-m1)) + 1e-6f);
    float ss = 0.0f;
    for (int p = 0; p < passes; ++p) {
        const int col = (p * cz + rank) * MS_COLS + x * VEC;
        float part[VEC], v[VEC];
#pragma unroll
        for (int c = 0; c < VEC; ++c) {
            part[c] = 0.0f;
            v[c] = col + c < vd ? row[2 * Hd + h * vd + col + c] : 0.0f;
        }
        for (int e0 = y; e0 < d; e0 += AHEAD * ROWS) {
            if (p || e0 != y) load(col, e0);
#pragma unroll
            for (int u = 0; u < AHEAD; ++u) {
                const int e = e0 + u * ROWS;
                if (e >= d || col >= vd) break;
#pragma unroll
                for (int c = 0; c < VEC; ++c) {
                    st[u][c] = fmaf(keep, st[u][c], ks[e] * v[c]);
                    part[c] = fmaf(st[u][c], qs[e], part[c]);
                }
                if (!live) continue;
                if (VEC == 4) *(float4*)(gS + (size_t)e * vd + col) = make_float4(st[u][0], st[u][VEC > 1 ? 1 : 0], st[u][VEC > 2 ? 2 : 0], st[u][VEC > 3 ? 3 : 0]);
                else gS[(size_t)e * vd + col] = st[u][0];
            }
        }
        if (VEC == 4) {                                         // the four rows that a warp holds of a column
#pragma unroll
            for (int c = 0; c < VEC; ++c) {
                part[c] += __shfl_xor_sync(0xffffffffu, part[c], 8);
                part[c] += __shfl_xor_sync(0xffffffffu, part[c], 16);
            }
            if ((threadIdx.x & 31) < 8) *(float4*)(red + (threadIdx.x >> 5) * MS_COLS + x * 4) = make_float4(part[0], part[VEC > 1 ? 1 : 0], part[VEC > 2 ? 2 : 0], part[VEC > 3 ? 3 : 0]);
        } else {
            red[y * MS_COLS + x] = part[0];
        }
        __syncthreads();
        if (threadIdx.x < MS_COLS) {
            float o = 0.0f;
#pragma unroll
            for (int r = 0; r < PARTS; ++r) o += red[r * MS_COLS + threadIdx.x];
            o *= inv_den;
            oc[p * MS_COLS + threadIdx.x] = o;
            ss = fmaf(o, o, ss);                                // columns beyond vd hold zeros
        }
        if (p + 1 < passes) __syncthreads();
    }
    if (threadIdx.x < 32) ss = sp_warp_sum(ss);
    float sum = 0.0f;
    if (cz > 1) {
        cluster_wait();
        if ((int)threadIdx.x < cz) store_peer_f32(&ssq[rank], threadIdx.x, ss);
        cluster_arrive();                                       // every CTA has read n and m and sent its squares
        cluster_wait();
        for (int c = 0; c < cz; ++c) sum += ssq[c];
    } else {
        if (threadIdx.x == 0) ssq[0] = ss;
        __syncthreads();
        sum = ssq[0];
    }
    const float f = 1.0f / sqrtf(sum / (float)vd + a.eps);
    if (live) {
        for (int p = 0; p < passes; ++p) {
            const int col = (p * cz + rank) * MS_COLS + threadIdx.x;
            if (threadIdx.x >= MS_COLS || col >= vd) break;
            if (p) {
                gate = g[col];
                weight = sp_ld_dt(a.nw, a.w_dt, (size_t)h * vd + col);
            }
            sp_st_dt(a.out, a.out_dt, (size_t)t * Hv + (size_t)h * vd + col, oc[p * MS_COLS + threadIdx.x] * f * weight / (1.0f + expf(-gate)));
        }
        if (rank == 0) {
            for (int e = threadIdx.x; e < d; e += 256) gn[e] = fmaf(keep, gn[e], ks[e]);
            if (threadIdx.x == 0) gn[d] = m1;
        }
    }
}

long long up4(long long n) { return (n + 3) / 4 * 4; }

}  // namespace

// Whether a prompt step with these operands can run on the tensor cores (bfloat16 outputs, 16-byte pieces everywhere).
SP_API int sp_mlstm_tc_supported(const void* proj, int ld, const void* nw, int w_dt, const float* state, const void* out, int out_dt, int d, int vd) {
    return out_dt == SP_DT_BF16 && w_dt == SP_DT_F32 && (((uintptr_t)state) & 15) == 0 && d % 8 == 0 && vd % 8 == 0 && ld % 4 == 0 &&
           ((((uintptr_t)proj | (uintptr_t)nw | (uintptr_t)out) & 15) == 0);
}
SP_API int sp_mlstm_chunk_tokens(int tensor_cores) { return tensor_cores ? TK : MC; }

// floats of scratch a prompt step needs
SP_API long long sp_mlstm_scratch_floats(int n_chunks, int T, int H, int d, int vd) {
    const long long vc = up4(vd + 1), HT = up4((long long)H * T);
    return 7 * HT + up4((long long)H * n_chunks) + up4((long long)n_chunks * H * d * vc) + (long long)T * H * vc;
}

// mode 0: a prompt step (``scratch``, ``n_chunks`` chunks of sp_mlstm_chunk_tokens(0)); 1: a decode step, one token per
// sequence; 2: a prompt step on the tensor cores (chunks of sp_mlstm_chunk_tokens(1))
SP_API int sp_mlstm(const float* proj, int ld, const void* ib, const void* fb, const void* nw, int w_dt, float* S, float* nm,
                    int n_slots, void* out, int out_dt, const int* seq_start, const int* seq_slot, int B, int T, int n_chunks,
                    int H, int d, int vd, float cap, float eps, float* scratch, int mode, int* status, cudaStream_t stream) {
    if (B <= 0 || T <= 0) return 0;
    if (H <= 0 || d <= 0 || vd <= 0 || H > 65535 || B > 65535) SP_FAIL("mlstm: sizes %d sequences, %d heads of %d x %d", B, H, d, vd);
    if (!(cap > 0.0f)) SP_FAIL("mlstm: the gates' cap must be positive");
    if (ld < 2 * H * (d + vd + 1)) SP_FAIL("mlstm: rows of %d numbers are too short", ld);
    MlArgs a{};
    a.proj = proj; a.ld = ld; a.ib = ib; a.fb = fb; a.nw = nw; a.w_dt = w_dt; a.S = S; a.nm = nm; a.n_slots = n_slots;
    a.out = out; a.out_dt = out_dt; a.seq_start = seq_start; a.seq_slot = seq_slot;
    a.B = B; a.T = T; a.H = H; a.d = d; a.vd = vd; a.n_chunks = n_chunks; a.cap = cap; a.eps = eps; a.status = status;
    if (mode == 1) {
        int cz = (vd + MS_COLS - 1) / MS_COLS;
        cz = cz >= 8 ? 8 : cz >= 4 ? 4 : cz >= 2 ? 2 : 1;
        const int passes = (vd + MS_COLS * cz - 1) / (MS_COLS * cz);
        const bool vec = vd % 4 == 0 && ((uintptr_t)S & 15) == 0;
        const size_t smem = ((size_t)2 * up4(d) + (size_t)(8 + passes) * MS_COLS) * sizeof(float);
        if (smem > 48 * 1024) SP_FAIL("mlstm (step): heads of %d x %d are beyond this kernel's range", d, vd);
        if (vec) SP_CHECK_CALL("mlstm_step", sp_launch_cluster(mlstm_step_kernel<4>, dim3(cz, H, B), dim3(256), smem, stream, -cz, a, cz));
        else SP_CHECK_CALL("mlstm_step", sp_launch_cluster(mlstm_step_kernel<1>, dim3(cz, H, B), dim3(256), smem, stream, -cz, a, cz));
        SP_CHECK_LAUNCH("mlstm_step");
        return 0;
    }
    if (!scratch || ((uintptr_t)scratch & 15)) SP_FAIL("mlstm: a prompt step needs scratch that starts on 16 bytes");
    if (mode == 2 && !sp_mlstm_tc_supported(proj, ld, nw, w_dt, S, out, out_dt, d, vd)) SP_FAIL("mlstm: the tensor-core form does not take these operands");
    const long long HT = up4((long long)H * T);
    a.vc = (int)up4(vd + 1);
    float* p = scratch;
    a.a2 = (float2*)p; p += 2 * HT;
    a.M2 = (float2*)p; p += 2 * HT;
    a.r = p; p += HT;
    a.we = p; p += HT;
    a.em = p; p += HT;
    a.ce = p; p += up4((long long)H * n_chunks);
    a.cs = p; p += up4((long long)n_chunks * H * d * a.vc);
    a.raw = p;
    static SpPerDevice ready;
    const int smem = (2 * 64 * MP + 64 * 64) * (int)sizeof(float), sum_smem = TK * OT_LD * 4 + 1024, out_smem = 2 * OT_STAGE + 1024;
    if (!ready.done()) {
        if (cudaFuncSetAttribute(mlstm_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess ||
            cudaFuncSetAttribute(mlstm_sum_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, sum_smem) != cudaSuccess ||
            cudaFuncSetAttribute(mlstm_out_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, out_smem) != cudaSuccess)
            SP_FAIL("mlstm: cannot raise the shared memory limit");
        ready.mark();
    }
    const dim3 scan_grid(B, H, (d * a.vc + 255) / 256);
    if (mode == 2) {
        const int cb = (vd + 255) / 256, eb = (d + TK - 1) / TK;
        SP_CHECK_CALL("mlstm_gates", sp_launch_dependent(mlstm_gates_kernel<TK>, dim3(B, H), dim3(MG_WARPS * 32), 0, stream, a));
        SP_CHECK_CALL("mlstm_sum_tc", sp_launch_dependent(mlstm_sum_tc_kernel, dim3(n_chunks, H, cb * eb), dim3(256), (size_t)sum_smem, stream, a));
        SP_CHECK_CALL("mlstm_scan", sp_launch_dependent(mlstm_scan_packed_kernel, dim3(B, H, (d * (a.vc / 4) + 127) / 128), dim3(128), 0, stream, a, TK));
        SP_CHECK_CALL("mlstm_out_tc", sp_launch_dependent(mlstm_out_tc_kernel, dim3(n_chunks, H, cb), dim3(OT_THREADS), (size_t)out_smem, stream, a));
        if (cb > 1) {
            mlstm_finish_kernel<<<dim3(T, H), 128, 0, stream>>>(a);
            SP_CHECK_LAUNCH("mlstm_finish");
        }
        return 0;
    }
    SP_CHECK_CALL("mlstm_gates", sp_launch_dependent(mlstm_gates_kernel<MC>, dim3(B, H), dim3(MG_WARPS * 32), 0, stream, a));
    const int nb = (vd + 64) / 64, eb = (d + 63) / 64;
    mlstm_sum_kernel<<<dim3(n_chunks, H, nb * eb), 256, 0, stream>>>(a);
    SP_CHECK_LAUNCH("mlstm_sum");
    SP_CHECK_CALL("mlstm_scan", sp_launch_dependent(mlstm_scan_kernel, scan_grid, dim3(256), 0, stream, a, MC));
    mlstm_out_kernel<<<dim3(n_chunks, H, nb), 256, smem, stream>>>(a);
    SP_CHECK_LAUNCH("mlstm_out");
    mlstm_finish_kernel<<<dim3(T, H), 128, 0, stream>>>(a);
    SP_CHECK_LAUNCH("mlstm_finish");
    return 0;
}
