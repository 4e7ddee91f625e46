// The real-gated linear recurrent unit behind a short causal convolution (a recurrent block's second branch).
//
// A projected row (32-bit) is [y: W | x: W], without the biases. Per channel c, at position p of a sequence:
//
//   u_p = β_c + Σ_k κ_c,k · (x_{p−taps+1+k} + b_c)              nothing (zero, not the bias) before the sequence's start
//   r = σ(R_b u_b + ρ),  i = σ(I_b u_b + ι)                     square matrices over equal parts u_b of the row
//   log a = −d_c · r,   S_p = a S_{p−1} + sqrt(1 − a²) · i ⊙ u_p,   out = S ⊙ gelu(y + b') · mult
//
// with d_c > 0 the channel's decay (made once from its weight). The state S and the last ``taps`` inputs x + b are kept
// per slot in 32-bit. The inputs are a ring: the input of position p stands in row p mod taps. A step reads rows
// p−1 … p−taps+1 and writes row p, which nobody reads in that step, so blocks that share inputs need no order.
//
//   rglru_chunk_*     prompts: the convolution feeds the two gate products (tensor cores with u as the sum of two bfloat16
//                     numbers, so that its rounding is 2⁻¹⁷: tcgen05 for parts of 128 or 256 channels, else mma.sync; or
//                     FFMA), the recurrence of each chunk of 64 (32) tokens runs from zero (a sequence's first chunk: from
//                     its state) and leaves per token (Π a, S), per chunk its end
//   rglru_scan        the chunks' start states one after another
//   rglru_finish      S = Π a · S_start + S_from_zero, times gelu(y); a sequence's last chunk leaves the state and the inputs
//   rglru_step        one token per sequence: all of it in one launch, the gate matrices streamed once per eight sequences
//
// Everything is 32-bit except the operands of the tensor-core products; the output is rounded once, on the store. A
// token's sums run in an order fixed by its row, whatever else is in the step.
#include "common.cuh"
#include "flash_common.cuh"
#include "tcgen05.cuh"

SP_API const char* sp_rglru_last_error() { return sp_error_text; }
SP_DEFINE_RANGE_API(rglru)

namespace {

constexpr int RG_CHUNK = 64;        // tokens of a block (and of a chunk, but for the tcgen05 kernel)
constexpr int RG_COLS = 64;         // channels of a block
constexpr int RG_SEGS = 4;          // a chunk's tokens are shared by four threads per channel
constexpr int RG_SEG = RG_CHUNK / RG_SEGS;

struct RgArgs {
    const float* proj; int ld;                      // [T][ld], y at 0, x at W
    const float* yb; const float* xb;               // [W]
    const float* conv; const float* convb;          // [W][taps], [W]
    const void* ra; const void* ri; int g_dt;       // [parts][size][size], rows = outputs
    const float* rab; const float* rib;             // [W]
    const float* decay;                             // [W]
    float* ring; float* state; int n_slots;         // [slots][taps][W], [slots][W]
    const int* seq_start; const int* seq_slot; const int* positions;
    float2* av; float2* cells;                      // [T][W] (Π a, S from zero); [chunks][W] a chunk's (Π a, S)
    float* starts;                                  // [chunks][W] the state in front of a chunk
    void* out; int out_dt;                          // [T][W]
    int T, B, W, taps, parts, size;
    float mult;
    int chunk;                                      // tokens of a chunk (what a cell stands for)
};

// Where a piece of a step's tokens stands.
struct RgPlace { int s, t0, n, first, pos0, slot; };

// the x-th piece of ``tokens`` tokens of the step's sequences
__device__ __forceinline__ bool rg_place(const RgArgs& a, int tokens, int x, RgPlace& pl) {
    for (int s = 0; s < a.B; ++s) {
        const int first = a.seq_start[s], cnt = a.seq_start[s + 1] - first;
        const int nc = (cnt + tokens - 1) / tokens;
        if (x < nc) {
            pl.s = s;
            pl.t0 = first + x * tokens;
            pl.n = min(tokens, cnt - x * tokens);
            pl.first = first;
            pl.pos0 = a.positions[first];
            pl.slot = a.seq_slot[s];
            return pl.slot >= 0 && pl.slot < a.n_slots;
        }
        x -= nc;
    }
    return false;
}

// The same for a block that takes pieces x in rising order: the sequence it stands in is remembered.
struct RgWalk {
    int s = -1, base = 0, nc = 0, first = 0, cnt = 0, pos0 = 0, slot = -1;
    __device__ __forceinline__ bool place(const RgArgs& a, int tokens, int x, RgPlace& pl) {
        while (x >= base + nc) {
            if (++s >= a.B) { s = a.B - 1; return false; }
            base += nc;
            first = a.seq_start[s];
            cnt = a.seq_start[s + 1] - first;
            nc = (cnt + tokens - 1) / tokens;
            pos0 = a.positions[first];
            slot = a.seq_slot[s];
        }
        pl.s = s; pl.first = first; pl.pos0 = pos0; pl.slot = slot;
        pl.t0 = first + (x - base) * tokens;
        pl.n = min(tokens, first + cnt - pl.t0);
        return slot >= 0 && slot < a.n_slots;
    }
};

// x + b of channel c at token ``t``: from the step's own rows, from the ring for the tokens before the step's first, or
// nothing before the sequence's start. There is no branch around the load, so that the loads of many tokens are under way
// together: the address is always one of the step's rows or of the ring's (a convolution of one tap never looks back).
__device__ __forceinline__ float rg_input(const RgArgs& a, const RgPlace& pl, int t, int c, float bias) {
    const bool here = t >= pl.first;
    const int p = pl.pos0 + (t - pl.first);
    const float* src = here ? a.proj + (size_t)t * a.ld + a.W + c
                            : a.ring + ((size_t)pl.slot * a.taps + (p >= 0 ? p % a.taps : 0)) * a.W + c;
    const float v = __ldg(src);
    return here ? v + bias : p >= 0 ? v : 0.0f;
}

// u of channel c for RG_SEG tokens from t; tokens at t_end or beyond get 0 (rows at the end stand in for those behind it).
template <int TAPS>
__device__ __forceinline__ void rg_conv(const RgArgs& a, const RgPlace& pl, int t, int t_end, int c, float (&u)[RG_SEG]) {
    const float bias = a.xb[c], beta = a.convb[c];
    if constexpr (TAPS > 0) {
        float x[RG_SEG + TAPS - 1], w[TAPS];
#pragma unroll
        for (int i = 0; i < RG_SEG + TAPS - 1; ++i) x[i] = rg_input(a, pl, min(t + i - (TAPS - 1), t_end - 1), c, bias);
#pragma unroll
        for (int k = 0; k < TAPS; ++k) w[k] = a.conv[(size_t)c * TAPS + k];
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) {
            float v = beta;
#pragma unroll
            for (int k = 0; k < TAPS; ++k) v = fmaf(w[k], x[i + k], v);
            u[i] = v;
        }
    } else {
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) u[i] = beta;
        for (int k = 0; k < a.taps; ++k) {
            const float w = a.conv[(size_t)c * a.taps + k];
#pragma unroll
            for (int i = 0; i < RG_SEG; ++i) u[i] = fmaf(w, rg_input(a, pl, min(t + i - (a.taps - 1) + k, t_end - 1), c, bias), u[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < RG_SEG; ++i) if (t + i >= t_end) u[i] = 0.0f;
}

__device__ __forceinline__ float rg_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// (decay of the step, what enters the state) of one token and channel from the gates' pre-activations
__device__ __forceinline__ void rg_gates(float zr, float zi, float u, float decay, float& d, float& v) {
    const float la = -decay * rg_sigmoid(zr);
    const float below = expm1f(la);                  // a − 1: exact where a is near 1, and a state remembers a's error for
    d = 1.0f + below;                                // thousands of tokens
    v = sqrtf(-below * (2.0f + below)) * rg_sigmoid(zi) * u;      // 1 − a² = −(a − 1)(a + 1)
}

// The same for the tensor-core kernels, whose gates come from operands of sixteen bits: the hardware's approximations (a few
// units in the last place). a − 1 keeps its relative accuracy near a = 1, where the state's memory lies: the power series
// of e^x − 1 for x > −0.3 (its next term is below 2⁻²⁷ of the sum there).
__device__ __forceinline__ float rg_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rg_sigmoid_fast(float z) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(1.0f + rg_ex2(-1.4426950408889634f * z)));
    return y;
}
__device__ __forceinline__ void rg_gates_fast(float zr, float zi, float u, float decay, float& d, float& v) {
    const float x = -decay * rg_sigmoid_fast(zr);
    float series = fmaf(x, 1.0f / 5040.0f, 1.0f / 720.0f);
    series = fmaf(x, series, 1.0f / 120.0f);
    series = fmaf(x, series, 1.0f / 24.0f);
    series = fmaf(x, series, 1.0f / 6.0f);
    series = fmaf(x, series, 0.5f);
    series = fmaf(x * x, series, x);
    const float below = x > -0.3f ? series : rg_ex2(1.4426950408889634f * x) - 1.0f;
    d = 1.0f + below;
    float root;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(root) : "f"(-below * (2.0f + below)));
    v = root * rg_sigmoid_fast(zi) * u;
}

constexpr int RG_GLD = RG_COLS + 2;                  // row of the gates' pre-activations in shared memory

// The block's recurrence from the gates' pre-activations G [2][64 tokens][RG_GLD]. Thread = (16 tokens, channel).
// ``u_of(row, i)``: u of token ``row`` of the chunk (the thread's i-th). FAST: rg_gates_fast. (No branch per token: the
// tokens' gates are computed side by side; a token behind the end keeps the state.)
template <bool FAST, typename U>
__device__ __forceinline__ void rg_block_scan(const RgArgs& a, const RgPlace& pl, int chunk, int c, bool c_ok, const float* G,
                                              float2 (*seg_end)[RG_COLS], U&& u_of) {
    const int cc = threadIdx.x & (RG_COLS - 1), seg = threadIdx.x / RG_COLS;
    const int t = pl.t0 + seg * RG_SEG, t_end = pl.t0 + pl.n;
    float A[RG_SEG], S[RG_SEG];
    float Ap = 1.0f, Sp = 0.0f;
    if (c_ok) {
        const float rb = a.rab[c], ib = a.rib[c], dec = a.decay[c];
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) {
            const int row = seg * RG_SEG + i;
            const float zr = G[row * RG_GLD + cc] + rb, zi = G[(RG_CHUNK + row) * RG_GLD + cc] + ib;
            if (FAST) rg_gates_fast(zr, zi, u_of(row, i), dec, A[i], S[i]);
            else rg_gates(zr, zi, u_of(row, i), dec, A[i], S[i]);
        }
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) {
            const float d = t + i < t_end ? A[i] : 1.0f, v = t + i < t_end ? S[i] : 0.0f;
            Sp = fmaf(d, Sp, v);
            Ap *= d;
            A[i] = Ap;
            S[i] = Sp;
        }
    }
    seg_end[seg][cc] = make_float2(Ap, Sp);
    __syncthreads();
    if (!c_ok) return;
    // a sequence's first chunk begins with its state (and nothing is left for the finish to bring in)
    const bool begins = pl.t0 == pl.first;
    float A0 = begins ? 0.0f : 1.0f, S0 = begins ? a.state[(size_t)pl.slot * a.W + c] : 0.0f;
    for (int j = 0; j < seg; ++j) {
        const float2 e = seg_end[j][cc];
        S0 = fmaf(e.x, S0, e.y);
        A0 *= e.x;
    }
#pragma unroll
    for (int i = 0; i < RG_SEG; ++i)
        if (t + i < t_end) a.av[(size_t)(t + i) * a.W + c] = make_float2(A0 * A[i], fmaf(A[i], S0, S[i]));
    if (seg == RG_SEGS - 1) a.cells[(size_t)chunk * a.W + c] = make_float2(A0 * Ap, fmaf(Ap, S0, Sp));
}

// ---------------------------------------------------------------- u for the tensor-core kernels
constexpr int RM_TOK = 8;                            // a thread makes u of two neighbouring channels for this many tokens

// The inputs of a convolution of TAPS taps over RM_TOK tokens of channels c and c + 1 (c even, rows on 8-byte boundaries), asked
// for by ``fetch`` and used by ``make``; rows at the end of the chunk stand in for those behind it.
template <int TAPS>
struct RgConv2 {
    static constexpr int BACK = TAPS > 0 ? TAPS - 1 : 0, N = RM_TOK + BACK;
    float2 x[N];

    __device__ __forceinline__ float2 load(const float* p) const { return __ldg((const float2*)p); }
    __device__ __forceinline__ void fetch(const RgArgs& a, const RgPlace& pl, int t, int t_end, int c) {
        if constexpr (TAPS > 0) {
            const float* row = a.proj + (size_t)t * a.ld + a.W + c;
            const int last = t_end - 1 - t;
#pragma unroll
            for (int i = 0; i < RM_TOK; ++i) x[BACK + i] = load(row + (size_t)min(i, last) * a.ld);
#pragma unroll
            for (int i = 0; i < BACK; ++i) {
                const int tt = t - BACK + i, p = pl.pos0 + (tt - pl.first);
                if (tt >= pl.first) x[i] = load(a.proj + (size_t)tt * a.ld + a.W + c);
                else if (p >= 0) x[i] = load(a.ring + ((size_t)pl.slot * TAPS + p % TAPS) * a.W + c);
                else x[i] = make_float2(0.0f, 0.0f);
            }
        }
    }

    // u of the tokens; tokens at t_end or beyond get 0. ``weight(k)``: both channels' tap k, then (TAPS) β, then (TAPS + 1) b
    template <typename W2>
    __device__ __forceinline__ void make(const RgArgs& a, const RgPlace& pl, int t, int t_end, int c, float2 (&u)[RM_TOK], W2&& weight) {
        const int c1 = c + 1;
        if constexpr (TAPS > 0) {
            const float2 beta = weight(TAPS), bias = weight(TAPS + 1);
            float2 w[TAPS];
#pragma unroll
            for (int k = 0; k < TAPS; ++k) w[k] = weight(k);
#pragma unroll
            for (int i = 0; i < N; ++i)
                if (i >= BACK || t - BACK + i >= pl.first) { x[i].x += bias.x; x[i].y += bias.y; }
#pragma unroll
            for (int i = 0; i < RM_TOK; ++i) {
                float2 v = beta;
#pragma unroll
                for (int k = 0; k < TAPS; ++k) { v.x = fmaf(w[k].x, x[i + k].x, v.x); v.y = fmaf(w[k].y, x[i + k].y, v.y); }
                u[i] = v;
            }
        } else {
            const float2 beta = make_float2(a.convb[c], a.convb[c1]), bias = make_float2(a.xb[c], a.xb[c1]);
#pragma unroll
            for (int i = 0; i < RM_TOK; ++i) u[i] = beta;
            for (int k = 0; k < a.taps; ++k) {
                const float2 w = make_float2(a.conv[(size_t)c * a.taps + k], a.conv[(size_t)c1 * a.taps + k]);
                float2 in[RM_TOK];
#pragma unroll
                for (int i = 0; i < RM_TOK; ++i) {
                    const int tt = min(t + i - (a.taps - 1) + k, t_end - 1);
                    in[i] = make_float2(rg_input(a, pl, tt, c, bias.x), rg_input(a, pl, tt, c1, bias.y));
                }
#pragma unroll
                for (int i = 0; i < RM_TOK; ++i) { u[i].x = fmaf(w.x, in[i].x, u[i].x); u[i].y = fmaf(w.y, in[i].y, u[i].y); }
            }
        }
#pragma unroll
        for (int i = 0; i < RM_TOK; ++i) if (t + i >= t_end) u[i] = make_float2(0.0f, 0.0f);
    }
};

template <int TAPS>
__device__ __forceinline__ float2 rg_conv_weight(const RgArgs& a, int c, int k) {
    if (k == TAPS) return make_float2(a.convb[c], a.convb[c + 1]);
    if (k == TAPS + 1) return make_float2(a.xb[c], a.xb[c + 1]);
    return make_float2(a.conv[(size_t)c * TAPS + k], a.conv[(size_t)(c + 1) * TAPS + k]);
}

// ---------------------------------------------------------------- gate products on mma.sync (parts of any multiple of 8)
constexpr int RM_BK = 64;
constexpr int RM_LD = RM_BK + 8;
constexpr int RM_A = RG_CHUNK * RM_LD;               // elements of one A buffer (high or low part)
constexpr int RM_B = 2 * RG_COLS * RM_LD;            // r and i rows
constexpr int RM_STAGE = 2 * RM_A + RM_B;
constexpr int RM_SMEM = 2 * RM_STAGE * 2;            // two stages of bfloat16
static_assert(2 * RG_CHUNK * RG_GLD * 4 <= RM_STAGE * 2, "the pre-activations lie over one stage");
static_assert(RM_BK == RG_COLS, "a block's own channels are one block of K");

template <int TAPS>
__global__ void __launch_bounds__(256)
rglru_chunk_mma_kernel(RgArgs a, int col_tiles) {
    extern __shared__ __align__(16) unsigned char rm_smem[];
    __shared__ float2 seg_end[RG_SEGS][RG_COLS];
    sp_allow_dependents();
    sp_wait_for_predecessor();
    RgPlace pl;
    if (!rg_place(a, RG_CHUNK, blockIdx.y, pl)) return;
    const int part = blockIdx.x / col_tiles, own = blockIdx.x % col_tiles, n0 = own * RG_COLS;
    const int size = a.size;
    __nv_bfloat16* sm = (__nv_bfloat16*)rm_smem;
    const __nv_bfloat16* wr = (const __nv_bfloat16*)a.ra + (size_t)part * size * size;
    const __nv_bfloat16* wi = (const __nv_bfloat16*)a.ri + (size_t)part * size * size;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t_end = pl.t0 + pl.n;
    const int nk = (size + RM_BK - 1) / RM_BK;
    // the blocks of K in order from the one behind the block's own channels: its own come last, so that their u is still in
    // shared memory when the gates meet it
    auto block_of = [&](int i) { const int kb = own + 1 + i; return kb < nk ? kb : kb - nk; };

    auto load_b = [&](int i) {
        __nv_bfloat16* B = sm + (i & 1) * RM_STAGE + 2 * RM_A;
        const int k0 = block_of(i) * RM_BK;
        // 2 x 64 rows of 64 numbers: 1,024 pieces of 16 bytes
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const int e = threadIdx.x + q * 256, g = e >> 9, row = (e >> 3) & 63, k8 = (e & 7) * 8;
            const int n = n0 + row, k = k0 + k8;
            __nv_bfloat16* dst = B + (g * RG_COLS + row) * RM_LD + k8;
            if (n < size && k < size) cp_async16(smem_u32(dst), (g ? wi : wr) + (size_t)n * size + k);
            else *(uint4*)dst = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
    // two channels per lane, eight tokens per warp; a block's inputs are asked for while the block before is multiplied
    const int row0 = warp * RM_TOK, t = pl.t0 + row0;
    RgConv2<TAPS> cv;
    auto fetch_a = [&](int i) {
        const int k = block_of(i) * RM_BK + 2 * lane;
        if (k < size && t < t_end) cv.fetch(a, pl, t, t_end, part * size + k);          // (the part's size is a multiple of 8)
    };
    auto make_a = [&](int i) {
        __nv_bfloat16* Ah = sm + (i & 1) * RM_STAGE;
        __nv_bfloat16* Al = Ah + RM_A;
        const int k = block_of(i) * RM_BK + 2 * lane;
        float2 u[RM_TOK];
        if (k < size && t < t_end) cv.make(a, pl, t, t_end, part * size + k, u, [&](int w) { return rg_conv_weight<TAPS>(a, part * size + k, w); });
        else {
#pragma unroll
            for (int r = 0; r < RM_TOK; ++r) u[r] = make_float2(0.0f, 0.0f);
        }
#pragma unroll
        for (int r = 0; r < RM_TOK; ++r) {
            const __nv_bfloat162 hi = __floats2bfloat162_rn(u[r].x, u[r].y);
            const float2 back = __bfloat1622float2(hi);
            *(__nv_bfloat162*)(Ah + (row0 + r) * RM_LD + 2 * lane) = hi;
            *(__nv_bfloat162*)(Al + (row0 + r) * RM_LD + 2 * lane) = __floats2bfloat162_rn(u[r].x - back.x, u[r].y - back.y);
        }
    };
    const int mi = warp & 3, gate = warp >> 2;       // a warp: 16 tokens x all 64 columns of one gate
    float acc[8][4] = {};
    load_b(0);
    fetch_a(0);
    for (int i = 0; i < nk; ++i) {
        make_a(i);
        if (i + 1 < nk) fetch_a(i + 1);
        cp_async_wait<0>();
        __syncthreads();                             // block i is complete; every warp is done with block i - 1
        if (i + 1 < nk) load_b(i + 1);
        const __nv_bfloat16* Ah = sm + (i & 1) * RM_STAGE;
        const __nv_bfloat16* Al = Ah + RM_A;
        const __nv_bfloat16* B = Ah + 2 * RM_A + gate * RG_COLS * RM_LD;
#pragma unroll
        for (int k16 = 0; k16 < RM_BK / 16; ++k16) {
            uint32_t h[4], l[4];
            const int ao = (mi * 16 + (lane & 15)) * RM_LD + k16 * 16 + (lane >> 4) * 8;
            ldmatrix_x4(smem_u32(Ah + ao), h[0], h[1], h[2], h[3]);
            ldmatrix_x4(smem_u32(Al + ao), l[0], l[1], l[2], l[3]);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(smem_u32(B + (np * 16 + (lane & 7) + (lane >> 4) * 8) * RM_LD + k16 * 16 + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
                mma_bf16(acc[2 * np], l, b0, b1);
                mma_bf16(acc[2 * np + 1], l, b2, b3);
                mma_bf16(acc[2 * np], h, b0, b1);
                mma_bf16(acc[2 * np + 1], h, b2, b3);
            }
        }
    }
    // the pre-activations [gate][token][RG_GLD] over the stage that the last block did not use; all warps are done with it
    // since they met in front of the last block's products
    float* G = (float*)(sm + (nk & 1) * RM_STAGE);
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int row = gate * RG_CHUNK + mi * 16 + (lane >> 2) + 8 * half;
            *(float2*)(G + row * RG_GLD + nt * 8 + (lane & 3) * 2) = make_float2(acc[nt][2 * half], acc[nt][2 * half + 1]);
        }
    __syncthreads();
    const __nv_bfloat16* Ah = sm + ((nk - 1) & 1) * RM_STAGE;
    const int cc = threadIdx.x & (RG_COLS - 1);
    rg_block_scan<true>(a, pl, blockIdx.y, part * size + n0 + cc, n0 + cc < size, G, seg_end, [&](int row, int) {
        return __bfloat162float(Ah[row * RM_LD + cc]) + __bfloat162float(Ah[RM_A + row * RM_LD + cc]);
    });
}

// ---------------------------------------------------------------- the same on tcgen05, turned round (parts of 128 and 256)
// The gate matrices' rows are the M of tcgen05.mma and the tokens its N, so that a channel is a lane of tensor memory and the
// recurrence runs along its columns: no exchange between threads. A CTA keeps 128 channels' rows of both gates (all of K) in
// shared memory and walks chunks of 32 tokens:
//   warp 0        one thread fetches the rows once by TMA (128-byte swizzle), ahead of the predecessor's end
//   warp 1        one thread issues the products of a chunk: for each gate 64 columns, the high parts of u and the low parts,
//                 whose sums meet in the registers (K-major operands)
//   warps 2-9     the convolution: u of the part's channels as two bfloat16 numbers, in the swizzled layout, two buffers; a
//                 warp makes 8 tokens of half the blocks of K, and the next block's inputs are on their way meanwhile
//   warps 10-17   two groups take the chunks in turn, thread = channel: u of its own channel into tensor memory beside the
//                 accumulator (the buffer is then free), gates from there, the recurrence, (Π a, S) out
// Two accumulators (r high | r low | i high | i low, 32 columns each) let the products of a chunk run under the recurrence of the one before. Every
// wait is bounded; one that runs out records a code, every role falls through to the common exit, tensor memory is freed.
constexpr int RT_ROWS = 128;                         // channels of a CTA
constexpr int RT_CHUNK = 32;                         // tokens of a chunk
constexpr int RT_THREADS = 18 * 32;
constexpr uint32_t RT_COLS = 512, RT_U = 256;        // tensor memory: two accumulators of 128 columns, from RT_U on 32 columns of u per group
template <int NKB> struct RtSmem {
    static constexpr int W_BOX = RT_ROWS * 128, U_BOX = 2 * RT_CHUNK * 128, LOW = RT_CHUNK * 128;
    static constexpr int W_BYTES = 2 * NKB * W_BOX, U_BYTES = NKB * U_BOX;           // [gate][block of K], [block of K][high | low rows]
    static constexpr int TAPS_AT = W_BYTES + 2 * U_BYTES;                            // [taps | β | b][the part's channels] float32
    static constexpr int total(int taps) { return TAPS_AT + (taps + 2) * NKB * 64 * 4 + 1024; }
};

template <int TAPS, int NKB>
__global__ void __launch_bounds__(RT_THREADS, 1)
rglru_chunk_tc_kernel(const __grid_constant__ CUtensorMap map_r, const __grid_constant__ CUtensorMap map_i, const RgArgs a,
                      int row_tiles, int walkers, int n_chunks, int* status) {
    using L = RtSmem<NKB>;
    static_assert(NKB % 2 == 0, "two halves of the convolution's warps share the blocks of K");
    extern __shared__ __align__(16) uint8_t rt_smem[];
    __shared__ __align__(8) uint64_t bar_w, bar_u_full[2], bar_u_free[2], bar_acc[2], bar_acc_free[2];
    __shared__ uint32_t tmem_slot;
    const uint32_t base = (smem_u32(rt_smem) + 1023u) & ~1023u;
    uint8_t* const base_ptr = rt_smem + (base - smem_u32(rt_smem));
    const uint32_t w_smem = base, u_smem = base + L::W_BYTES;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int tile_c = blockIdx.x % row_tiles, walker = blockIdx.x / row_tiles;
    const int c0 = tile_c * RT_ROWS, part = c0 / a.size, n0 = c0 - part * a.size;     // a part is one or two tiles
    if (threadIdx.x == 0) {
        mbar_init(smem_u32(&bar_w), 1);
        for (int b = 0; b < 2; ++b) {                     // arrivals by warp: eight of the convolution, four of a group
            mbar_init(smem_u32(&bar_u_full[b]), 8);
            mbar_init(smem_u32(&bar_u_free[b]), 4);
            mbar_init(smem_u32(&bar_acc[b]), 1);
            mbar_init(smem_u32(&bar_acc_free[b]), 4);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_u32(&tmem_slot)), "r"(RT_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    if (warp == 0 && lane == 0) {
        mbar_expect_tx(smem_u32(&bar_w), L::W_BYTES);
        for (int kb = 0; kb < NKB; ++kb) {
            tma_load_2d(w_smem + kb * L::W_BOX, &map_r, kb * 64, c0, smem_u32(&bar_w));
            tma_load_2d(w_smem + (NKB + kb) * L::W_BOX, &map_i, kb * 64, c0, smem_u32(&bar_w));
        }
    }
    // the convolution's weights of the part's channels (nobody's output either)
    float* const taps_smem = (float*)(base_ptr + L::TAPS_AT);
    for (int e = threadIdx.x; e < (TAPS + 2) * NKB * 64; e += RT_THREADS) {
        const int kk = e / (NKB * 64), cc = part * a.size + e % (NKB * 64);
        taps_smem[e] = kk < TAPS ? a.conv[(size_t)cc * TAPS + kk] : kk == TAPS ? a.convb[cc] : a.xb[cc];
    }
    __syncthreads();
    sp_allow_dependents();
    sp_wait_for_predecessor();

    if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(RT_ROWS, 2 * RT_CHUNK);
            bool ok = mbar_wait(smem_u32(&bar_w), 0, status, 141);
            uint32_t it = 0;
            RgPlace pl;
            RgWalk walk;
            for (int x = walker; x < n_chunks && ok; x += walkers) {
                if (!walk.place(a, RT_CHUNK, x, pl)) continue;
                const uint32_t buf = it & 1u, phase = (it >> 1) & 1u;
                ok = mbar_wait(smem_u32(&bar_acc_free[buf]), phase ^ 1u, status, 143) &&
                     mbar_wait(smem_u32(&bar_u_full[buf]), phase, status, 144);
                if (!ok) break;
                tc_fence_after();
#pragma unroll
                for (int gate = 0; gate < 2; ++gate)
#pragma unroll
                    for (int kb = 0; kb < NKB; ++kb) {
                        const uint64_t dw = umma_desc_sw128(w_smem + (gate * NKB + kb) * L::W_BOX);
                        const uint64_t du = umma_desc_sw128(u_smem + buf * L::U_BYTES + kb * L::U_BOX);
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            tc_mma_bf16(tmem + buf * 128u + (uint32_t)gate * 64u, dw + 2 * k, du + 2 * k, idesc, (kb | k) == 0 ? 0u : 1u);
                    }
                tc_commit(smem_u32(&bar_acc[buf]));
                ++it;
            }
        }
    } else if (warp >= 2 && warp < 10) {
        // eight tokens and half the blocks of K per warp, two channels of a block per lane
        const int row0 = ((warp - 2) & 3) * RM_TOK, kb0 = ((warp - 2) >> 2) * (NKB / 2);
        const int c = part * a.size + kb0 * 64 + 2 * lane;
        bool ok = true;
        uint32_t it = 0;
        RgPlace pl, ahead;
        RgConv2<TAPS> cur, nxt;                                      // the inputs that come next are asked for while one block is made
        int x = walker;
        RgWalk walk;
        auto find = [&](RgPlace& p) {                                // the next chunk that exists, from x on
            for (; x < n_chunks; x += walkers) if (walk.place(a, RT_CHUNK, x, p)) return true;
            return false;
        };
        bool have = find(pl), more = false;
        if (have && row0 < pl.n) cur.fetch(a, pl, pl.t0 + row0, pl.t0 + pl.n, c);
        int j = 0;
#pragma unroll 1
        while (have) {
            const bool last_j = j + 1 == NKB / 2;
            if (last_j) { x += walkers; more = find(ahead); }
            const RgPlace& np = last_j ? ahead : pl;
            const int nj = last_j ? 0 : j + 1;
            if ((!last_j || more) && row0 < np.n) nxt.fetch(a, np, np.t0 + row0, np.t0 + np.n, c + nj * 64);
            const uint32_t buf = it & 1u;
            if (j == 0) {
                ok = mbar_wait(smem_u32(&bar_u_free[buf]), ((it >> 1) & 1u) ^ 1u, status, 142);
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
            }
            float2 u[RM_TOK];
            if (row0 < pl.n) cur.make(a, pl, pl.t0 + row0, pl.t0 + pl.n, c + j * 64, u, [&](int w) {
                return *(const float2*)(taps_smem + w * NKB * 64 + (kb0 + j) * 64 + 2 * lane);
            });
            else {
#pragma unroll
                for (int r = 0; r < RM_TOK; ++r) u[r] = make_float2(0.0f, 0.0f);
            }
            uint8_t* hi_box = base_ptr + L::W_BYTES + buf * L::U_BYTES + (kb0 + j) * L::U_BOX + row0 * 128;      // row0 is a multiple of 8: row & 7 = r
#pragma unroll
            for (int r = 0; r < RM_TOK; ++r) {
                const uint32_t at = r * 128 + (((lane >> 2) ^ r) << 4) + (lane & 3) * 4;
                const __nv_bfloat162 hi = __floats2bfloat162_rn(u[r].x, u[r].y);
                const float2 back = __bfloat1622float2(hi);
                *(__nv_bfloat162*)(hi_box + at) = hi;
                *(__nv_bfloat162*)(hi_box + L::LOW + at) = __floats2bfloat162_rn(u[r].x - back.x, u[r].y - back.y);
            }
            if (last_j) {
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");      // the products read what these stores wrote
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&bar_u_full[buf]));
                ++it;
                pl = ahead;
                have = more;
            }
            j = nj;
            cur = nxt;
        }
    } else if (warp >= 10) {
        const uint32_t group = (uint32_t)(warp - 10) >> 2;           // takes every second chunk of this CTA
        const int q = warp & 3;                                      // lanes 32q … of tensor memory
        const int ch = q * 32 + lane, c = c0 + ch;
        const float rb = a.rab[c], ib = a.rib[c], dec = a.decay[c];
        const int k = (n0 + ch) & 63;
        const uint8_t* own = base_ptr + L::W_BYTES + group * L::U_BYTES + ((n0 + ch) >> 6) * L::U_BOX + (k & 7) * 2;
        bool ok = true;
        uint32_t it = 0;
        RgPlace pl;
        RgWalk walk;
        for (int x = walker; x < n_chunks && ok; x += walkers) {
            if (!walk.place(a, RT_CHUNK, x, pl)) continue;
            if ((it & 1u) != group) { ++it; continue; }
            const uint32_t phase = (it >> 1) & 1u;
            ++it;
            // (the convolution's own barrier too: this warp reads what those warps stored)
            ok = mbar_wait(smem_u32(&bar_u_full[group]), phase, status, 145) && mbar_wait(smem_u32(&bar_acc[group]), phase, status, 145);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            const uint32_t lanes = tmem + ((uint32_t)(q * 32) << 16), own_u = lanes + RT_U + group * RT_CHUNK;
            {
                uint32_t up[RT_CHUNK];                               // high part above, low part below
#pragma unroll
                for (int i = 0; i < RT_CHUNK; ++i) {
                    const uint8_t* p = own + i * 128 + (((k >> 3) ^ (i & 7)) << 4);
                    up[i] = ((uint32_t)*(const uint16_t*)p << 16) | *(const uint16_t*)(p + L::LOW);
                }
                tc_st_32x32(own_u, up);
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&bar_u_free[group]));
                tc_st_wait();
            }
            const int t = pl.t0, n = pl.n;
            const bool begins = t == pl.first;                       // a sequence's first chunk begins with its state
            float A = begins ? 0.0f : 1.0f, S = begins ? a.state[(size_t)pl.slot * a.W + c] : 0.0f;
            float2* av = a.av + (size_t)t * a.W + c;
            const uint32_t acc = lanes + group * 128u;
            // eight tokens at a time: their gates side by side (no branch per token), then the recurrence
#pragma unroll 1
            for (int h = 0; h < RT_CHUNK / 8; ++h) {
                uint32_t zr[8], zi[8], lr[8], li[8];
                tc_ld_32x8(acc + h * 8, zr);
                tc_ld_32x8(acc + 32 + h * 8, lr);
                tc_ld_32x8(acc + 64 + h * 8, zi);
                tc_ld_32x8(acc + 96 + h * 8, li);
                uint32_t up[8];
                tc_ld_32x8(own_u + h * 8, up);
                tc_ld_wait();
                if (h == RT_CHUNK / 8 - 1) {
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(smem_u32(&bar_acc_free[group]));
                }
                float d[8], v[8];
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    rg_gates_fast(__uint_as_float(zr[i]) + (__uint_as_float(lr[i]) + rb), __uint_as_float(zi[i]) + (__uint_as_float(li[i]) + ib),
                                  __uint_as_float(up[i] & 0xffff0000u) + __uint_as_float(up[i] << 16), dec, d[i], v[i]);
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    if (h * 8 + i < n) {
                        S = fmaf(d[i], S, v[i]);
                        A *= d[i];
                        av[(size_t)(h * 8 + i) * a.W] = make_float2(A, S);
                    }
                }
            }
            a.cells[(size_t)x * a.W + c] = make_float2(A, S);        // chunks are counted as cells are
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(RT_COLS) : "memory");
    }
}

// ---------------------------------------------------------------- the same with FFMA (32-bit operands, any sizes)
constexpr int RF_BK = 32;
constexpr int RF_LD = RG_CHUNK + 4;                  // rows of k, 64 tokens or columns each

template <int TAPS, typename TW>
__global__ void __launch_bounds__(256)
rglru_chunk_ffma_kernel(RgArgs a, int col_tiles) {
    __shared__ __align__(16) float buf[3 * RF_BK * RF_LD > 2 * RG_CHUNK * RG_GLD ? 3 * RF_BK * RF_LD : 2 * RG_CHUNK * RG_GLD];
    __shared__ float2 seg_end[RG_SEGS][RG_COLS];
    RgPlace pl;
    if (!rg_place(a, RG_CHUNK, blockIdx.y, pl)) return;
    const int part = blockIdx.x / col_tiles, n0 = (blockIdx.x % col_tiles) * RG_COLS;
    const int size = a.size;
    const TW* wr = (const TW*)a.ra + (size_t)part * size * size;
    const TW* wi = (const TW*)a.ri + (size_t)part * size * size;
    const int t_end = pl.t0 + pl.n;
    float* As = buf;                                 // [k][token]
    float* Bs = buf + RF_BK * RF_LD;                 // [gate][k][column]
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;      // 4 tokens x 4 columns x 2 gates
    float acc[2][4][4] = {};
    for (int k0 = 0; k0 < size; k0 += RF_BK) {
        if (threadIdx.x < RF_BK * RG_SEGS) {
            const int kk = threadIdx.x & (RF_BK - 1), seg = threadIdx.x / RF_BK;
            float u[RG_SEG];
            if (k0 + kk < size) rg_conv<TAPS>(a, pl, pl.t0 + seg * RG_SEG, t_end, part * size + k0 + kk, u);
            else {
#pragma unroll
                for (int i = 0; i < RG_SEG; ++i) u[i] = 0.0f;
            }
#pragma unroll
            for (int i = 0; i < RG_SEG; ++i) As[kk * RF_LD + seg * RG_SEG + i] = u[i];
        }
        for (int e = threadIdx.x; e < 2 * RG_COLS * RF_BK; e += 256) {
            const int kk = e % RF_BK, n = (e / RF_BK) % RG_COLS, g = e / (RF_BK * RG_COLS);
            Bs[(g * RF_BK + kk) * RF_LD + n] = (n0 + n < size && k0 + kk < size) ? sp_ld(g ? wi : wr, (size_t)(n0 + n) * size + k0 + kk) : 0.0f;
        }
        __syncthreads();
#pragma unroll 8
        for (int kk = 0; kk < RF_BK; ++kk) {
            const float4 x4 = *(const float4*)(As + kk * RF_LD + 4 * ty);
            const float x[4] = {x4.x, x4.y, x4.z, x4.w};
#pragma unroll
            for (int g = 0; g < 2; ++g) {
                const float4 b4 = *(const float4*)(Bs + (g * RF_BK + kk) * RF_LD + 4 * tx);
                const float b[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[g][i][j] = fmaf(x[i], b[j], acc[g][i][j]);
            }
        }
        __syncthreads();
    }
    float* G = buf;
#pragma unroll
    for (int g = 0; g < 2; ++g)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) G[(g * RG_CHUNK + 4 * ty + i) * RG_GLD + 4 * tx + j] = acc[g][i][j];
    __syncthreads();
    const int cc = threadIdx.x & (RG_COLS - 1), c = part * size + n0 + cc;
    float u[RG_SEG];
    if (n0 + cc < size) rg_conv<TAPS>(a, pl, pl.t0 + threadIdx.x / RG_COLS * RG_SEG, t_end, c, u);
    rg_block_scan<false>(a, pl, blockIdx.y, c, n0 + cc < size, G, seg_end, [&](int, int i) { return u[i]; });
}

// ---------------------------------------------------------------- start states of the chunks
// A block: 32 channels of one sequence; its eight warps compose a stretch of the chunks' ends each, then every warp knows
// where its stretch begins and writes its chunks' start states.
__global__ void __launch_bounds__(256) rglru_scan_kernel(RgArgs a) {
    __shared__ float2 stretch[8][32];
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int s = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
    int chunk = 0;
    for (int b = 0; b < s; ++b) chunk += (a.seq_start[b + 1] - a.seq_start[b] + a.chunk - 1) / a.chunk;
    const int n = (a.seq_start[s + 1] - a.seq_start[s] + a.chunk - 1) / a.chunk, per = (n + 7) / 8;
    const int x0 = min(n, warp * per), x1 = min(n, x0 + per);
    const bool ok = c < a.W && a.seq_slot[s] >= 0 && a.seq_slot[s] < a.n_slots;       // else nobody wrote the cells
    const float2* cell = a.cells + (size_t)chunk * a.W + c;
    float A = 1.0f, S = 0.0f;
    if (ok) {
#pragma unroll 8
        for (int x = x0; x < x1; ++x) {
            const float2 e = cell[(size_t)x * a.W];
            S = fmaf(e.x, S, e.y);
            A *= e.x;
        }
    }
    stretch[warp][lane] = make_float2(A, S);
    __syncthreads();
    if (!ok) return;
    S = 0.0f;                                        // the first chunk's cell holds the sequence's state already
    for (int w = 0; w < warp; ++w) { const float2 e = stretch[w][lane]; S = fmaf(e.x, S, e.y); }
    float* start = a.starts + (size_t)chunk * a.W + c;
#pragma unroll 8
    for (int x = x0; x < x1; ++x) {
        const float2 e = cell[(size_t)x * a.W];
        start[(size_t)x * a.W] = S;
        S = fmaf(e.x, S, e.y);
    }
}

// ---------------------------------------------------------------- outputs of a prompt step
constexpr int RN_ROWS = 4;                           // rows of a warp under way together
constexpr int RN_TOK = 32;                           // tokens of a block (a chunk is one or two blocks)
template <int VEC>
__global__ void __launch_bounds__(256) rglru_finish_kernel(RgArgs a) {
    sp_allow_dependents();
    sp_wait_for_predecessor();
    RgPlace pl;
    if (!rg_place(a, RN_TOK, blockIdx.y, pl)) return;
    const int lane = threadIdx.x & 31, row = threadIdx.x >> 5;
    const int c = (blockIdx.x * 32 + lane) * VEC;
    if (c >= a.W) return;
    int chunk = (pl.t0 - pl.first) / a.chunk;
    for (int b = 0; b < pl.s; ++b) chunk += (a.seq_start[b + 1] - a.seq_start[b] + a.chunk - 1) / a.chunk;
    if constexpr (VEC == 4) {
        float4 e0[RN_ROWS], e1[RN_ROWS], y[RN_ROWS];
#pragma unroll
        for (int k = 0; k < RN_ROWS; ++k) {
            const size_t t = pl.t0 + min(row + 8 * k, pl.n - 1), o = t * a.W + c;
            e0[k] = *(const float4*)(a.av + o);
            e1[k] = *(const float4*)(a.av + o + 2);
            y[k] = *(const float4*)(a.proj + t * a.ld + c);
        }
        const float4 start = *(const float4*)(a.starts + (size_t)chunk * a.W + c), yb = *(const float4*)(a.yb + c);
#pragma unroll
        for (int k = 0; k < RN_ROWS; ++k) {
            if (row + 8 * k >= pl.n) break;
            const size_t o = (size_t)(pl.t0 + row + 8 * k) * a.W + c;
            const float r0 = fmaf(e0[k].x, start.x, e0[k].y) * sp_gelu_tanh(y[k].x + yb.x) * a.mult;
            const float r1 = fmaf(e0[k].z, start.y, e0[k].w) * sp_gelu_tanh(y[k].y + yb.y) * a.mult;
            const float r2 = fmaf(e1[k].x, start.z, e1[k].y) * sp_gelu_tanh(y[k].z + yb.z) * a.mult;
            const float r3 = fmaf(e1[k].z, start.w, e1[k].w) * sp_gelu_tanh(y[k].w + yb.w) * a.mult;
            if (a.out_dt == SP_DT_F32) *(float4*)((float*)a.out + o) = make_float4(r0, r1, r2, r3);
            else {
                __nv_bfloat162 p0 = __floats2bfloat162_rn(r0, r1), p1 = __floats2bfloat162_rn(r2, r3);
                uint2 pk;
                pk.x = *(uint32_t*)&p0; pk.y = *(uint32_t*)&p1;
                *(uint2*)((__nv_bfloat16*)a.out + o) = pk;
            }
        }
        static_assert(RN_TOK == 8 * RN_ROWS, "eight warps share the block's rows");
    } else {
        const float start = a.starts[(size_t)chunk * a.W + c];
        for (int i = row; i < pl.n; i += 8) {
            const size_t t = pl.t0 + i, o = t * a.W + c;
            const float2 e = a.av[o];
            sp_st_dt(a.out, a.out_dt, o, fmaf(e.x, start, e.y) * sp_gelu_tanh(a.proj[t * a.ld + c] + a.yb[c]) * a.mult);
        }
    }
    if (pl.t0 + pl.n == a.seq_start[pl.s + 1] && row == 0) {
        // the sequence's last block leaves the state and the last inputs (nothing of this launch reads either)
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
            const float2 e = a.cells[(size_t)chunk * a.W + c + j];
            a.state[(size_t)pl.slot * a.W + c + j] = fmaf(e.x, a.starts[(size_t)chunk * a.W + c + j], e.y);
        }
        if (a.taps > 1)
            for (int t = max(pl.first, pl.t0 + pl.n - a.taps); t < pl.t0 + pl.n; ++t)
#pragma unroll
                for (int j = 0; j < VEC; ++j)
                    a.ring[((size_t)pl.slot * a.taps + a.positions[t] % a.taps) * a.W + c + j] =
                        a.proj[(size_t)t * a.ld + a.W + c + j] + a.xb[c + j];
    }
}

// ---------------------------------------------------------------- one token per sequence
// A block: 8 channels of one part, a warp each, for up to TB sequences. Its u of the whole part waits in shared memory (the
// blocks of a part each make it, from the same ring rows); a warp streams its channel's two gate rows (the first eight weights
// per lane are asked for before the kernel waits for its predecessor: weights are nobody's output) and holds 2 x TB sums,
// which meet across the lanes so that every pair of lanes ends with one of them.
constexpr int RS_ROWS = 8;

// eight neighbouring weights
__device__ __forceinline__ void rs_load8(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 q = *(const uint4*)p;
    const __nv_bfloat162* h = (const __nv_bfloat162*)&q;
#pragma unroll
    for (int j = 0; j < 4; ++j) { const float2 v = __bfloat1622float2(h[j]); f[2 * j] = v.x; f[2 * j + 1] = v.y; }
}
__device__ __forceinline__ void rs_load8(const float* p, float (&f)[8]) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const float4 v = *(const float4*)(p + 4 * j);
        f[4 * j] = v.x; f[4 * j + 1] = v.y; f[4 * j + 2] = v.z; f[4 * j + 3] = v.w;
    }
}

template <typename TW, int TB, int TAPS>
__global__ void __launch_bounds__(256) rglru_step_kernel(RgArgs a, int row_tiles, int vec) {
    extern __shared__ __align__(16) float rs_u[];    // [TB][size rounded up to 4]
    __shared__ int s_tok[TB], s_slot[TB], s_pos[TB];
    const int part = blockIdx.x / row_tiles, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n = (blockIdx.x % row_tiles) * RS_ROWS + warp;         // this warp's channel within the part
    const int size = a.size, ld = (size + 3) & ~3;
    const bool row_ok = n < size;
    const TW* rr = (const TW*)a.ra + ((size_t)part * size + (row_ok ? n : 0)) * size;
    const TW* ir = (const TW*)a.ri + ((size_t)part * size + (row_ok ? n : 0)) * size;
    float fr[8], fi[8];
    if (vec && lane * 8 < size) { rs_load8(rr + lane * 8, fr); rs_load8(ir + lane * 8, fi); }
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int s0 = blockIdx.y * TB, nb = min(TB, a.B - s0);
    if (threadIdx.x < TB) {
        int t = 0, slot = -1, pos = 0;
        if ((int)threadIdx.x < nb) { t = a.seq_start[s0 + threadIdx.x]; slot = a.seq_slot[s0 + threadIdx.x]; pos = a.positions[t]; }
        s_tok[threadIdx.x] = t;
        s_slot[threadIdx.x] = slot >= 0 && slot < a.n_slots ? slot : -1;
        s_pos[threadIdx.x] = pos;
    }
    __syncthreads();
    // what the end of this channel needs is asked for now: lane 2b finishes sequence b
    const int c = part * size + n, b = (lane >> 1) & (TB - 1);
    const bool live = row_ok && (lane & 1) == 0 && lane < 2 * TB && b < nb && s_slot[b] >= 0;
    float S = 0.0f, y = 0.0f, x = 0.0f;
    if (live) {
        S = a.state[(size_t)s_slot[b] * a.W + c];
        y = a.proj[(size_t)s_tok[b] * a.ld + c] + a.yb[c];
        x = a.proj[(size_t)s_tok[b] * a.ld + a.W + c] + a.xb[c];
    }
    const int taps = TAPS > 0 ? TAPS : a.taps;
    for (int k = threadIdx.x; k < size; k += 256) {
        const int ck = part * size + k;
        const float bias = a.xb[ck], beta = a.convb[ck];
        if constexpr (TAPS > 0) {
            float w[TAPS], in[TB][TAPS];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j] = a.conv[(size_t)ck * TAPS + j];
#pragma unroll
            for (int i = 0; i < TB; ++i) {
                const int slot = max(s_slot[i], 0), pos = s_pos[i];
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {                 // position pos − (TAPS − 1) + j: always an address of the ring
                    const int p = pos - (TAPS - 1) + j;
                    const float v = a.ring[((size_t)slot * TAPS + (p + TAPS) % TAPS) * a.W + ck];
                    in[i][j] = p >= 0 ? v : 0.0f;
                }
                in[i][TAPS - 1] = a.proj[(size_t)s_tok[i] * a.ld + a.W + ck] + bias;
            }
#pragma unroll
            for (int i = 0; i < TB; ++i) {
                float u = beta;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) u = fmaf(w[j], in[i][j], u);
                rs_u[i * ld + k] = u;
            }
        } else {
            for (int i = 0; i < nb; ++i) {
                RgPlace pl;
                pl.first = s_tok[i]; pl.pos0 = s_pos[i]; pl.slot = max(s_slot[i], 0);
                float u = beta;
                for (int j = 0; j < taps; ++j)
                    u = fmaf(a.conv[(size_t)ck * taps + j], rg_input(a, pl, s_tok[i] - (taps - 1) + j, ck, bias), u);
                rs_u[i * ld + k] = u;
            }
        }
    }
    __syncthreads();
    if (!row_ok) return;
    float v[2 * TB];
#pragma unroll
    for (int i = 0; i < 2 * TB; ++i) v[i] = 0.0f;
    if (vec) {
        for (int k = lane * 8; k < size; k += 256) {
            if (k != lane * 8) { rs_load8(rr + k, fr); rs_load8(ir + k, fi); }
#pragma unroll
            for (int i = 0; i < TB; ++i) {
                if (i >= nb) break;
                const float4 u0 = *(const float4*)(rs_u + i * ld + k), u1 = *(const float4*)(rs_u + i * ld + k + 4);
                const float u[8] = {u0.x, u0.y, u0.z, u0.w, u1.x, u1.y, u1.z, u1.w};
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    v[i] = fmaf(fr[j], u[j], v[i]);
                    v[TB + i] = fmaf(fi[j], u[j], v[TB + i]);
                }
            }
        }
    } else {
        for (int k = lane; k < size; k += 32) {
            const float r1 = sp_ld(rr, k), i1 = sp_ld(ir, k);
#pragma unroll
            for (int i = 0; i < TB; ++i) {
                if (i >= nb) break;
                const float u = rs_u[i * ld + k];
                v[i] = fmaf(r1, u, v[i]);
                v[TB + i] = fmaf(i1, u, v[TB + i]);
            }
        }
    }
    // halve the values a lane holds while halving the lanes they are spread over
    int held = 2 * TB, off = 16;
#pragma unroll
    for (int step = 0; step < 4; ++step) {
        if (held > 1) {
            held >>= 1;
            const bool upper = (lane & off) != 0;
#pragma unroll
            for (int i = 0; i < TB; ++i) {
                if (i < held) {
                    const float keep = upper ? v[held + i] : v[i], give = upper ? v[i] : v[held + i];
                    v[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
                }
            }
            off >>= 1;
        }
    }
    for (; off > 0; off >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
    // value index (r: b, i: TB + b) = the lane's upper bits; bring r and i of a sequence together and to lane 2b
    const int span = 32 / (2 * TB);                          // lanes that hold the same value
    const float zr = __shfl_sync(0xffffffffu, v[0], b * span), zi = __shfl_sync(0xffffffffu, v[0], (TB + b) * span);
    if (live) {
        float d, in;
        rg_gates(zr + a.rab[c], zi + a.rib[c], rs_u[b * ld + n], a.decay[c], d, in);
        S = fmaf(d, S, in);
        a.state[(size_t)s_slot[b] * a.W + c] = S;
        if (taps > 1) a.ring[((size_t)s_slot[b] * taps + s_pos[b] % taps) * a.W + c] = x;
        sp_st_dt(a.out, a.out_dt, (size_t)s_tok[b] * a.W + c, S * sp_gelu_tanh(y) * a.mult);
    }
}

int check(const RgArgs& a) {
    if (a.W <= 0 || a.parts <= 0 || a.size <= 0 || a.parts * a.size != a.W) SP_FAIL("rglru: %d parts of %d do not make a width of %d", a.parts, a.size, a.W);
    if (a.taps < 1) SP_FAIL("rglru: the convolution needs at least one tap, got %d", a.taps);
    if (a.ld < 2 * a.W) SP_FAIL("rglru: rows of %d numbers are too short for two branches of %d", a.ld, a.W);
    if (a.g_dt != SP_DT_F32 && a.g_dt != SP_DT_BF16) SP_FAIL("rglru: unsupported dtype code %d", a.g_dt);
    return 0;
}

// A gate's stack of matrices [rows, size] as boxes of 128 rows x 64 columns. Maps are kept: the weights never move.
int gate_map(CUtensorMap* map, const void* ptr, int rows, int size) {
    typedef CUresult (*Encode)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                               const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    struct Slot { const void* ptr; int rows, size; CUtensorMap map; };
    static Slot kept[256];
    Slot& slot = kept[((uintptr_t)ptr >> 8) % 256];
    if (slot.ptr == ptr && slot.rows == rows && slot.size == size) {
        *map = slot.map;
        return 0;
    }
    static Encode encode = nullptr;
    if (!encode) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult found;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &found) != cudaSuccess || found != cudaDriverEntryPointSuccess)
            SP_FAIL("rglru: the driver does not offer cuTensorMapEncodeTiled");
        encode = (Encode)p;
    }
    cuuint64_t dims[2] = {(cuuint64_t)size, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)size * 2};
    cuuint32_t box[2] = {64, RT_ROWS}, steps[2] = {1, 1};
    const CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, steps,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) SP_FAIL("rglru: cuTensorMapEncodeTiled failed with code %d", (int)r);
    slot.ptr = ptr; slot.rows = rows; slot.size = size; slot.map = *map;
    return 0;
}

template <int TAPS, int NKB>
int launch_tc(const CUtensorMap& mr, const CUtensorMap& mi, const RgArgs& a, int n_chunks, int* status, cudaStream_t stream) {
    static SpPerDevice ready;
    if (!ready.done()) {
        if (cudaFuncSetAttribute(rglru_chunk_tc_kernel<TAPS, NKB>, cudaFuncAttributeMaxDynamicSharedMemorySize, RtSmem<NKB>::total(TAPS)) != cudaSuccess)
            SP_FAIL("rglru: cannot reserve %d bytes of shared memory", RtSmem<NKB>::total(TAPS));
        ready.mark();
    }
    const int row_tiles = a.W / RT_ROWS, sms = sp_sm_count();
    int walkers = sms / row_tiles;
    walkers = walkers < 1 ? 1 : walkers > n_chunks ? n_chunks : walkers;
    SP_CHECK_CALL("rglru_chunk", sp_launch_dependent(rglru_chunk_tc_kernel<TAPS, NKB>, dim3(row_tiles * walkers), dim3(RT_THREADS),
                                                     (size_t)RtSmem<NKB>::total(TAPS), stream, mr, mi, a, row_tiles, walkers, n_chunks, status));
    return 0;
}

bool takes_tc(int g_dt, int size, int tensor_cores) { return tensor_cores && g_dt == SP_DT_BF16 && (size == 128 || size == 256); }
bool in_pairs(const RgArgs& a) { return (a.ld & 1) == 0 && (a.W & 1) == 0 && (((uintptr_t)a.proj | (uintptr_t)a.ring) & 7) == 0; }

}  // namespace

// Tokens of a chunk (what one row of ``cells`` stands for) when sp_rglru_chunked runs these operands.
SP_API int sp_rglru_chunk_tokens(int g_dt, int size, int tensor_cores) { return takes_tc(g_dt, size, tensor_cores) ? RT_CHUNK : RG_CHUNK; }
SP_API int sp_rglru_finish_tokens() { return RN_TOK; }

// A step of prompts or portions. ``av``: [T][W] pairs of floats, ``cells``: [n_chunks][W] pairs, ``starts``: [n_chunks][W]
// floats; ``n_chunks``: the sequences' chunks of sp_rglru_chunk_tokens tokens, ``n_blocks``: of sp_rglru_finish_tokens.
SP_API int sp_rglru_chunked(const float* proj, int ld, const float* yb, const float* xb, const float* conv, const float* convb,
                            const void* ra, const void* ri, int g_dt, const float* rab, const float* rib, const float* decay,
                            float* ring, float* state, int n_slots, const int* seq_start, const int* seq_slot,
                            const int* positions, float* av, float* cells, float* starts, int n_chunks, int n_blocks, void* out,
                            int out_dt, int T, int B, int W, int taps, int parts, float mult, int tensor_cores, int* status,
                            cudaStream_t stream) {
    if (T <= 0 || B <= 0 || n_chunks <= 0) return 0;
    RgArgs a{proj, ld, yb, xb, conv, convb, ra, ri, g_dt, rab, rib, decay, ring, state, n_slots, seq_start, seq_slot, positions,
             (float2*)av, (float2*)cells, starts, out, out_dt, T, B, W, taps, parts, parts > 0 ? W / parts : 0, mult, RG_CHUNK};
    if (check(a)) return 1;
    if (n_chunks > 65535 || n_blocks > 65535) SP_FAIL("rglru: %d chunks are too many for one launch", n_blocks);
    const bool aligned = (((uintptr_t)ra | (uintptr_t)ri) & 15) == 0;
    const bool tc = takes_tc(g_dt, a.size, tensor_cores);
    const int col_tiles = (a.size + RG_COLS - 1) / RG_COLS;
    const dim3 grid(parts * col_tiles, n_chunks);
    if (tc) {
        a.chunk = RT_CHUNK;
        if (!aligned || !in_pairs(a)) SP_FAIL("rglru: the gate matrices must start on a 16-byte boundary, rows and ring on 8-byte ones");
        CUtensorMap mr, mi;
        if (gate_map(&mr, ra, W, a.size) || gate_map(&mi, ri, W, a.size)) return 1;
        if (a.size == 256 ? (taps == 4 ? launch_tc<4, 4>(mr, mi, a, n_chunks, status, stream) : launch_tc<0, 4>(mr, mi, a, n_chunks, status, stream))
                          : (taps == 4 ? launch_tc<4, 2>(mr, mi, a, n_chunks, status, stream) : launch_tc<0, 2>(mr, mi, a, n_chunks, status, stream)))
            return 1;
    } else if (tensor_cores && g_dt == SP_DT_BF16 && a.size % 8 == 0 && aligned && in_pairs(a)) {
        static SpPerDevice ready;
        if (!ready.done()) {
            if (cudaFuncSetAttribute(rglru_chunk_mma_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, RM_SMEM) != cudaSuccess ||
                cudaFuncSetAttribute(rglru_chunk_mma_kernel<0>, cudaFuncAttributeMaxDynamicSharedMemorySize, RM_SMEM) != cudaSuccess)
                SP_FAIL("rglru: cannot reserve %d bytes of shared memory", RM_SMEM);
            ready.mark();
        }
        if (taps == 4) SP_CHECK_CALL("rglru_chunk", sp_launch_dependent(rglru_chunk_mma_kernel<4>, grid, dim3(256), (size_t)RM_SMEM, stream, a, col_tiles));
        else SP_CHECK_CALL("rglru_chunk", sp_launch_dependent(rglru_chunk_mma_kernel<0>, grid, dim3(256), (size_t)RM_SMEM, stream, a, col_tiles));
    } else {
        if (g_dt == SP_DT_BF16) {
            if (taps == 4) rglru_chunk_ffma_kernel<4, __nv_bfloat16><<<grid, 256, 0, stream>>>(a, col_tiles);
            else rglru_chunk_ffma_kernel<0, __nv_bfloat16><<<grid, 256, 0, stream>>>(a, col_tiles);
        } else {
            if (taps == 4) rglru_chunk_ffma_kernel<4, float><<<grid, 256, 0, stream>>>(a, col_tiles);
            else rglru_chunk_ffma_kernel<0, float><<<grid, 256, 0, stream>>>(a, col_tiles);
        }
        SP_CHECK_LAUNCH("rglru_chunk (FFMA)");
    }
    SP_CHECK_CALL("rglru_scan", sp_launch_dependent(rglru_scan_kernel, dim3((W + 31) / 32, B), dim3(256), 0, stream, a));
    const bool vec = W % 4 == 0 && ld % 4 == 0 && (((uintptr_t)proj | (uintptr_t)av | (uintptr_t)starts | (uintptr_t)yb | (uintptr_t)out) & 15) == 0;
    if (vec) SP_CHECK_CALL("rglru_finish", sp_launch_dependent(rglru_finish_kernel<4>, dim3((W + 127) / 128, n_blocks), dim3(256), 0, stream, a));
    else SP_CHECK_CALL("rglru_finish", sp_launch_dependent(rglru_finish_kernel<1>, dim3((W + 31) / 32, n_blocks), dim3(256), 0, stream, a));
    return 0;
}

// A step with one token per sequence.
SP_API int sp_rglru_step(const float* proj, int ld, const float* yb, const float* xb, const float* conv, const float* convb,
                         const void* ra, const void* ri, int g_dt, const float* rab, const float* rib, const float* decay,
                         float* ring, float* state, int n_slots, const int* seq_start, const int* seq_slot, const int* positions,
                         void* out, int out_dt, int B, int W, int taps, int parts, float mult, cudaStream_t stream) {
    if (B <= 0) return 0;
    RgArgs a{proj, ld, yb, xb, conv, convb, ra, ri, g_dt, rab, rib, decay, ring, state, n_slots, seq_start, seq_slot, positions,
             nullptr, nullptr, nullptr, out, out_dt, B, B, W, taps, parts, parts > 0 ? W / parts : 0, mult, 1};
    if (check(a)) return 1;
    const int row_tiles = (a.size + RS_ROWS - 1) / RS_ROWS, ldu = (a.size + 3) & ~3;
    const int vec = a.size % 8 == 0 && (((uintptr_t)ra | (uintptr_t)ri) & 15) == 0;
    // as many sequences per block as their inputs leave room for in shared memory
    const int tb = (size_t)8 * ldu * 4 <= 48 * 1024 ? 8 : 1;
    const size_t smem = (size_t)tb * ldu * 4;
    if (smem > 48 * 1024) SP_FAIL("rglru: parts of %d channels are beyond the step kernel's shared memory", a.size);
    const int groups = (B + tb - 1) / tb;
    if (groups > 65535) SP_FAIL("rglru: %d sequences are too many for one launch", B);
    const dim3 grid(parts * row_tiles, groups);
#define RS_LAUNCH(TW, TB, TAPS) SP_CHECK_CALL("rglru_step", sp_launch_dependent(rglru_step_kernel<TW, TB, TAPS>, grid, dim3(256), smem, stream, a, row_tiles, vec))
    if (g_dt == SP_DT_BF16) {
        if (tb == 8 && taps == 4) RS_LAUNCH(__nv_bfloat16, 8, 4);
        else if (tb == 8) RS_LAUNCH(__nv_bfloat16, 8, 0);
        else RS_LAUNCH(__nv_bfloat16, 1, 0);
    } else {
        if (tb == 8 && taps == 4) RS_LAUNCH(float, 8, 4);
        else if (tb == 8) RS_LAUNCH(float, 8, 0);
        else RS_LAUNCH(float, 1, 0);
    }
#undef RS_LAUNCH
    return 0;
}
