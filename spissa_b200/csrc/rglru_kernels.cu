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
//   rglru_chunk_*     prompts: blocks of 64 tokens x 64 channels of one part. The convolution feeds the two gate products
//                     (tensor cores with u as the sum of two bfloat16 numbers, so that its rounding is 2⁻¹⁷; or FFMA), the
//                     block's recurrence runs from zero and leaves per token (Π a, S), per block its end
//   rglru_scan        the blocks' start states one after another; the last inputs into the ring
//   rglru_finish      S = Π a · S_start + S_from_zero, times gelu(y)
//   rglru_step        one token per sequence: all of it in one launch, the gate matrices streamed once per eight sequences
//
// Everything is 32-bit except the operands of the tensor-core products; the output is rounded once, on the store. A
// token's sums run in an order fixed by its row, whatever else is in the step.
#include "common.cuh"
#include "flash_common.cuh"

SP_API const char* sp_rglru_last_error() { return sp_error_text; }
SP_DEFINE_RANGE_API(rglru)

namespace {

constexpr int RG_CHUNK = 64;        // tokens of a chunk
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
    float2* av; float2* cells;                      // [T][W] (Π a, S from zero); [chunks][W] a chunk's (Π a, S), then (start, ·)
    void* out; int out_dt;                          // [T][W]
    int T, B, W, taps, parts, size;
    float mult;
};

__device__ __forceinline__ float rg_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

__device__ __forceinline__ bool rg_chunk_of(const int* seq_start, int B, int x, int& s, int& t0, int& n) {
    for (s = 0; s < B; ++s) {
        const int first = seq_start[s], cnt = seq_start[s + 1] - first;
        const int nc = (cnt + RG_CHUNK - 1) / RG_CHUNK;
        if (x < nc) {
            t0 = first + x * RG_CHUNK;
            n = min(RG_CHUNK, cnt - x * RG_CHUNK);
            return true;
        }
        x -= nc;
    }
    return false;
}

// x + b of channel c at token ``t`` of a sequence whose step begins at token ``first`` with position ``pos0``: from the
// step's own rows, from the ring, or nothing before the sequence's start.
__device__ __forceinline__ float rg_input(const RgArgs& a, int t, int first, int pos0, int slot, int c, float bias) {
    if (t >= first) return a.proj[(size_t)t * a.ld + a.W + c] + bias;
    const int p = pos0 + (t - first);
    return p < 0 ? 0.0f : a.ring[((size_t)slot * a.taps + p % a.taps) * a.W + c];
}

// Where a chunk's block stands.
struct RgPlace { int s, t0, n, first, pos0, slot; };

// u of channel c for RG_SEG tokens from t; tokens at t_end or beyond get 0.
template <int TAPS>
__device__ __forceinline__ void rg_conv(const RgArgs& a, const RgPlace& pl, int t, int t_end, int c, float (&u)[RG_SEG]) {
    const float bias = a.xb[c], beta = a.convb[c];
    if (TAPS > 0) {
        float x[RG_SEG + (TAPS > 0 ? TAPS - 1 : 0)], w[TAPS > 0 ? TAPS : 1];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) w[k] = a.conv[(size_t)c * TAPS + k];
#pragma unroll
        for (int i = 0; i < RG_SEG + TAPS - 1; ++i) {
            const int tt = t + i - (TAPS - 1);
            x[i] = tt < t_end ? rg_input(a, tt, pl.first, pl.pos0, pl.slot, c, bias) : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) {
            float v = beta;
#pragma unroll
            for (int k = 0; k < TAPS; ++k) v = fmaf(w[k], x[i + k], v);
            u[i] = t + i < t_end ? v : 0.0f;
        }
    } else {
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) u[i] = beta;
        for (int k = 0; k < a.taps; ++k) {
            const float w = a.conv[(size_t)c * a.taps + k];
#pragma unroll
            for (int i = 0; i < RG_SEG; ++i) {
                const int tt = t + i - (a.taps - 1) + k;
                if (t + i < t_end) u[i] = fmaf(w, rg_input(a, tt, pl.first, pl.pos0, pl.slot, c, bias), u[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) if (t + i >= t_end) u[i] = 0.0f;
    }
}

// (decay of the step, what enters the state) of one token and channel from the gates' pre-activations
__device__ __forceinline__ void rg_gates(float zr, float zi, float u, float decay, float& d, float& v) {
    const float la = -decay * rg_sigmoid(zr);
    const float below = expm1f(la);                  // a − 1: exact where a is near 1, and a state remembers a's error for
    d = 1.0f + below;                                // thousands of tokens (expf's last bit leans to one side there)
    v = sqrtf(-below * (2.0f + below)) * rg_sigmoid(zi) * u;      // 1 − a² = −(a − 1)(a + 1)
}

constexpr int RG_GLD = RG_COLS + 2;                  // row of the gates' pre-activations in shared memory

// The block's recurrence from zero, from the gates' pre-activations G [2][64 tokens][RG_GLD]. Thread = (16 tokens, channel).
template <int TAPS>
__device__ __forceinline__ void rg_block_scan(const RgArgs& a, const RgPlace& pl, int chunk, int c, bool c_ok, const float* G,
                                              float2 (*seg_end)[RG_COLS]) {
    const int cc = threadIdx.x & (RG_COLS - 1), seg = threadIdx.x / RG_COLS;
    const int t = pl.t0 + seg * RG_SEG, t_end = pl.t0 + pl.n;
    float A[RG_SEG], S[RG_SEG];
    float Ap = 1.0f, Sp = 0.0f;
    if (c_ok) {
        float u[RG_SEG];
        rg_conv<TAPS>(a, pl, t, t_end, c, u);
        const float rb = a.rab[c], ib = a.rib[c], dec = a.decay[c];
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) {
            float d = 1.0f, v = 0.0f;
            if (t + i < t_end) {
                const int row = seg * RG_SEG + i;
                rg_gates(G[row * RG_GLD + cc] + rb, G[(RG_CHUNK + row) * RG_GLD + cc] + ib, u[i], dec, d, v);
            }
            Sp = fmaf(d, Sp, v);
            Ap *= d;
            A[i] = Ap;
            S[i] = Sp;
        }
    }
    seg_end[seg][cc] = make_float2(Ap, Sp);
    __syncthreads();
    if (!c_ok) return;
    float A0 = 1.0f, S0 = 0.0f;
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

__device__ __forceinline__ bool rg_place(const RgArgs& a, int chunk, RgPlace& pl) {
    if (!rg_chunk_of(a.seq_start, a.B, chunk, pl.s, pl.t0, pl.n)) return false;
    pl.first = a.seq_start[pl.s];
    pl.pos0 = a.positions[pl.first];
    pl.slot = a.seq_slot[pl.s];
    return pl.slot >= 0 && pl.slot < a.n_slots;
}

// ---------------------------------------------------------------- gate products on the tensor cores
constexpr int RM_BK = 64;
constexpr int RM_LD = RM_BK + 8;
constexpr int RM_A = RG_CHUNK * RM_LD;               // elements of one A buffer (high or low part)
constexpr int RM_B = 2 * RG_COLS * RM_LD;            // r and i rows
constexpr int RM_STAGE = 2 * RM_A + RM_B;
constexpr int RM_SMEM = 2 * RM_STAGE * 2;            // two stages of bfloat16
static_assert(2 * RG_CHUNK * RG_GLD * 4 <= RM_SMEM, "the pre-activations lie over the stages");

template <int TAPS>
__global__ void __launch_bounds__(256)
rglru_chunk_mma_kernel(RgArgs a, int col_tiles) {
    extern __shared__ __align__(16) unsigned char rm_smem[];
    __shared__ float2 seg_end[RG_SEGS][RG_COLS];
    sp_allow_dependents();
    sp_wait_for_predecessor();
    RgPlace pl;
    if (!rg_place(a, blockIdx.y, pl)) return;
    const int part = blockIdx.x / col_tiles, n0 = (blockIdx.x % col_tiles) * RG_COLS;
    const int size = a.size;
    __nv_bfloat16* sm = (__nv_bfloat16*)rm_smem;
    const __nv_bfloat16* w[2] = {(const __nv_bfloat16*)a.ra + (size_t)part * size * size, (const __nv_bfloat16*)a.ri + (size_t)part * size * size};
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cc = threadIdx.x & (RG_COLS - 1), seg = threadIdx.x / RG_COLS;
    const int t_end = pl.t0 + pl.n;
    const int nk = (size + RM_BK - 1) / RM_BK;

    auto load_b = [&](int kb) {
        __nv_bfloat16* B = sm + (kb & 1) * RM_STAGE + 2 * RM_A;
        // 2 x 64 rows of 64 numbers: 1,024 pieces of 16 bytes
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = threadIdx.x + i * 256, g = e >> 9, row = (e >> 3) & 63, k8 = (e & 7) * 8;
            const int n = n0 + row, k = kb * RM_BK + k8;
            __nv_bfloat16* dst = B + (g * RG_COLS + row) * RM_LD + k8;
            if (n < size && k < size) cp_async16(smem_u32(dst), w[g] + (size_t)n * size + k);
            else *(uint4*)dst = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
    auto make_a = [&](int kb) {
        __nv_bfloat16* Ah = sm + (kb & 1) * RM_STAGE;
        __nv_bfloat16* Al = Ah + RM_A;
        float u[RG_SEG];
        const int k = kb * RM_BK + cc;
        if (k < size) rg_conv<TAPS>(a, pl, pl.t0 + seg * RG_SEG, t_end, part * size + k, u);
        else {
#pragma unroll
            for (int i = 0; i < RG_SEG; ++i) u[i] = 0.0f;
        }
#pragma unroll
        for (int i = 0; i < RG_SEG; ++i) {
            const __nv_bfloat16 hi = __float2bfloat16_rn(u[i]);
            Ah[(seg * RG_SEG + i) * RM_LD + cc] = hi;
            Al[(seg * RG_SEG + i) * RM_LD + cc] = __float2bfloat16_rn(u[i] - __bfloat162float(hi));
        }
    };
    const int mi = warp & 3, gate = warp >> 2;       // a warp: 16 tokens x all 64 columns of one gate
    float acc[8][4] = {};
    load_b(0);
    for (int kb = 0; kb < nk; ++kb) {
        make_a(kb);
        cp_async_wait<0>();
        __syncthreads();                             // block kb is complete; every warp is done with block kb - 1
        if (kb + 1 < nk) load_b(kb + 1);
        const __nv_bfloat16* Ah = sm + (kb & 1) * RM_STAGE;
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
                mma_bf16(acc[2 * np], h, b0, b1);
                mma_bf16(acc[2 * np + 1], l, b2, b3);
                mma_bf16(acc[2 * np + 1], h, b2, b3);
            }
        }
    }
    __syncthreads();
    float* G = (float*)rm_smem;                      // [gate][token][RG_GLD]
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int row = gate * RG_CHUNK + mi * 16 + (lane >> 2) + 8 * half;
            *(float2*)(G + row * RG_GLD + nt * 8 + (lane & 3) * 2) = make_float2(acc[nt][2 * half], acc[nt][2 * half + 1]);
        }
    __syncthreads();
    const int c = part * size + n0 + cc;
    rg_block_scan<TAPS>(a, pl, blockIdx.y, c, n0 + cc < size, G, seg_end);
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
    if (!rg_place(a, blockIdx.y, pl)) return;
    const int part = blockIdx.x / col_tiles, n0 = (blockIdx.x % col_tiles) * RG_COLS;
    const int size = a.size;
    const TW* w[2] = {(const TW*)a.ra + (size_t)part * size * size, (const TW*)a.ri + (size_t)part * size * size};
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
            Bs[(g * RF_BK + kk) * RF_LD + n] = (n0 + n < size && k0 + kk < size) ? sp_ld(w[g], (size_t)(n0 + n) * size + k0 + kk) : 0.0f;
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
    const int cc = threadIdx.x & (RG_COLS - 1);
    rg_block_scan<TAPS>(a, pl, blockIdx.y, part * size + n0 + cc, n0 + cc < size, G, seg_end);
}

// ---------------------------------------------------------------- start states; the inputs' ring
__global__ void __launch_bounds__(128) rglru_scan_kernel(RgArgs a) {
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int s = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (s >= a.B || c >= a.W) return;
    const int slot = a.seq_slot[s];
    if (slot < 0 || slot >= a.n_slots) return;
    int chunk = 0;
    for (int b = 0; b < s; ++b) chunk += (a.seq_start[b + 1] - a.seq_start[b] + RG_CHUNK - 1) / RG_CHUNK;
    const int first = a.seq_start[s], cnt = a.seq_start[s + 1] - first;
    const int n_chunks = (cnt + RG_CHUNK - 1) / RG_CHUNK;
    float S = a.state[(size_t)slot * a.W + c];
    float2* cell = a.cells + (size_t)chunk * a.W + c;
    for (int x0 = 0; x0 < n_chunks; x0 += 8) {
        float2 e[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (x0 + u < n_chunks) e[u] = cell[(size_t)(x0 + u) * a.W];          // eight cells in flight
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            if (x0 + u >= n_chunks) break;
            cell[(size_t)(x0 + u) * a.W].x = S;
            S = fmaf(e[u].x, S, e[u].y);
        }
    }
    a.state[(size_t)slot * a.W + c] = S;
    if (a.taps > 1) {
        const float bias = a.xb[c];
        for (int t = max(first, first + cnt - a.taps); t < first + cnt; ++t)
            a.ring[((size_t)slot * a.taps + a.positions[t] % a.taps) * a.W + c] = a.proj[(size_t)t * a.ld + a.W + c] + bias;
    }
}

// ---------------------------------------------------------------- outputs of a prompt step
template <int VEC>
__global__ void __launch_bounds__(256) rglru_finish_kernel(RgArgs a) {
    sp_allow_dependents();
    sp_wait_for_predecessor();
    RgPlace pl;
    if (!rg_place(a, blockIdx.y, pl)) return;
    const int lane = threadIdx.x & 31, row = threadIdx.x >> 5;
    const int c = (blockIdx.x * 32 + lane) * VEC;
    if (c >= a.W) return;
    float start[VEC], yb[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
        start[j] = a.cells[(size_t)blockIdx.y * a.W + c + j].x;
        yb[j] = a.yb[c + j];
    }
#pragma unroll 2
    for (int i = row; i < pl.n; i += 8) {
        const size_t t = pl.t0 + i, o = t * a.W + c;
        if (VEC == 4) {
            const float4 e0 = *(const float4*)(a.av + o), e1 = *(const float4*)(a.av + o + 2);
            const float4 y = *(const float4*)(a.proj + t * a.ld + c);
            const float r0 = fmaf(e0.x, start[0], e0.y) * sp_gelu_tanh(y.x + yb[0]) * a.mult;
            const float r1 = fmaf(e0.z, start[1 % VEC], e0.w) * sp_gelu_tanh(y.y + yb[1 % VEC]) * a.mult;
            const float r2 = fmaf(e1.x, start[2 % VEC], e1.y) * sp_gelu_tanh(y.z + yb[2 % VEC]) * a.mult;
            const float r3 = fmaf(e1.z, start[3 % VEC], e1.w) * sp_gelu_tanh(y.w + yb[3 % VEC]) * a.mult;
            if (a.out_dt == SP_DT_F32) *(float4*)((float*)a.out + o) = make_float4(r0, r1, r2, r3);
            else {
                __nv_bfloat162 p0 = __floats2bfloat162_rn(r0, r1), p1 = __floats2bfloat162_rn(r2, r3);
                uint2 pk;
                pk.x = *(uint32_t*)&p0; pk.y = *(uint32_t*)&p1;
                *(uint2*)((__nv_bfloat16*)a.out + o) = pk;
            }
        } else {
            const float2 e = a.av[o];
            sp_st_dt(a.out, a.out_dt, o, fmaf(e.x, start[0], e.y) * sp_gelu_tanh(a.proj[t * a.ld + c] + yb[0]) * a.mult);
        }
    }
}

// ---------------------------------------------------------------- one token per sequence
// A block: 16 channels of one part for up to TB sequences. Its u of the whole part waits in shared memory (the blocks of a
// part each make it, from the same ring rows); a warp streams a channel's two gate rows and holds 2 x TB sums, which
// meet across the lanes so that every pair of lanes ends with one of them.
constexpr int RS_ROWS = 16;

template <typename TW, int TB>
__global__ void __launch_bounds__(256) rglru_step_kernel(RgArgs a, int row_tiles, int vec) {
    extern __shared__ __align__(16) float rs_u[];    // [TB][size rounded up to 4]
    sp_allow_dependents();
    sp_wait_for_predecessor();
    const int part = blockIdx.x / row_tiles, n0 = (blockIdx.x % row_tiles) * RS_ROWS;
    const int s0 = blockIdx.y * TB, nb = min(TB, a.B - s0);
    const int size = a.size, ld = (size + 3) & ~3;
    for (int e = threadIdx.x; e < nb * size; e += 256) {
        const int b = e / size, k = e - b * size, c = part * size + k;
        const int t = a.seq_start[s0 + b], slot = a.seq_slot[s0 + b], pos = a.positions[t];
        float u = 0.0f;
        if (slot >= 0 && slot < a.n_slots) {
            const float bias = a.xb[c];
            u = a.convb[c];
            for (int j = 0; j < a.taps; ++j)
                u = fmaf(a.conv[(size_t)c * a.taps + j], rg_input(a, t - (a.taps - 1) + j, t, pos, slot, c, bias), u);
        }
        rs_u[b * ld + k] = u;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const TW* wr = (const TW*)a.ra + (size_t)part * size * size;
    const TW* wi = (const TW*)a.ri + (size_t)part * size * size;
    for (int n = n0 + warp; n < min(size, n0 + RS_ROWS); n += 8) {
        const int c = part * size + n;
        // what the end of this channel needs is asked for first: lane 2b (and 2b + 1) finishes sequence b
        const int b = (lane >> 1) & (TB - 1);
        const bool mine = lane < 2 * TB && b < nb;
        const int t = mine ? a.seq_start[s0 + b] : 0, slot = mine ? a.seq_slot[s0 + b] : -1;
        const bool live = mine && slot >= 0 && slot < a.n_slots;
        float S = 0.0f, y = 0.0f, x = 0.0f;
        if (live) {
            S = a.state[(size_t)slot * a.W + c];
            y = a.proj[(size_t)t * a.ld + c] + a.yb[c];
            x = a.proj[(size_t)t * a.ld + a.W + c] + a.xb[c];
        }
        float v[2 * TB];
#pragma unroll
        for (int i = 0; i < 2 * TB; ++i) v[i] = 0.0f;
        const TW* rr = wr + (size_t)n * size;
        const TW* ir = wi + (size_t)n * size;
        if (vec) {
            // eight neighbouring weights of each row per lane and turn
            for (int k = lane * 8; k < size; k += 256) {
                float fr[8], fi[8];
                if (sizeof(TW) == 2) {
                    const uint4 q = *(const uint4*)(rr + k), p = *(const uint4*)(ir + k);
                    const __nv_bfloat162* qq = (const __nv_bfloat162*)&q;
                    const __nv_bfloat162* pp = (const __nv_bfloat162*)&p;
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float2 f = __bfloat1622float2(qq[j]), g = __bfloat1622float2(pp[j]);
                        fr[2 * j] = f.x; fr[2 * j + 1] = f.y; fi[2 * j] = g.x; fi[2 * j + 1] = g.y;
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        const float4 f = *(const float4*)((const float*)rr + k + 4 * j), g = *(const float4*)((const float*)ir + k + 4 * j);
                        fr[4 * j] = f.x; fr[4 * j + 1] = f.y; fr[4 * j + 2] = f.z; fr[4 * j + 3] = f.w;
                        fi[4 * j] = g.x; fi[4 * j + 1] = g.y; fi[4 * j + 2] = g.z; fi[4 * j + 3] = g.w;
                    }
                }
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
                const float fr = sp_ld(rr, k), fi = sp_ld(ir, k);
#pragma unroll
                for (int i = 0; i < TB; ++i) {
                    if (i >= nb) break;
                    const float u = rs_u[i * ld + k];
                    v[i] = fmaf(fr, u, v[i]);
                    v[TB + i] = fmaf(fi, u, v[TB + i]);
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
        if (live && (lane & 1) == 0) {
            float d, in;
            rg_gates(zr + a.rab[c], zi + a.rib[c], rs_u[b * ld + n], a.decay[c], d, in);
            S = fmaf(d, S, in);
            a.state[(size_t)slot * a.W + c] = S;
            if (a.taps > 1) a.ring[((size_t)slot * a.taps + a.positions[t] % a.taps) * a.W + c] = x;
            sp_st_dt(a.out, a.out_dt, (size_t)t * a.W + c, S * sp_gelu_tanh(y) * a.mult);
        }
    }
}

int check(const RgArgs& a) {
    if (a.W <= 0 || a.parts <= 0 || a.size <= 0 || a.parts * a.size != a.W) SP_FAIL("rglru: %d parts of %d do not make a width of %d", a.parts, a.size, a.W);
    if (a.taps < 1) SP_FAIL("rglru: the convolution needs at least one tap, got %d", a.taps);
    if (a.ld < 2 * a.W) SP_FAIL("rglru: rows of %d numbers are too short for two branches of %d", a.ld, a.W);
    if (a.g_dt != SP_DT_F32 && a.g_dt != SP_DT_BF16) SP_FAIL("rglru: unsupported dtype code %d", a.g_dt);
    return 0;
}

}  // namespace

SP_API int sp_rglru_chunk_tokens() { return RG_CHUNK; }

// A step of prompts or portions. ``av``: [T][W] pairs of floats, ``cells``: [n_chunks][W] pairs.
SP_API int sp_rglru_chunked(const float* proj, int ld, const float* yb, const float* xb, const float* conv, const float* convb,
                            const void* ra, const void* ri, int g_dt, const float* rab, const float* rib, const float* decay,
                            float* ring, float* state, int n_slots, const int* seq_start, const int* seq_slot,
                            const int* positions, float* av, float* cells, int n_chunks, void* out, int out_dt, int T, int B, int W,
                            int taps, int parts, float mult, int tensor_cores, cudaStream_t stream) {
    if (T <= 0 || B <= 0 || n_chunks <= 0) return 0;
    RgArgs a{proj, ld, yb, xb, conv, convb, ra, ri, g_dt, rab, rib, decay, ring, state, n_slots, seq_start, seq_slot, positions,
             (float2*)av, (float2*)cells, out, out_dt, T, B, W, taps, parts, parts > 0 ? W / parts : 0, mult};
    if (check(a)) return 1;
    if (n_chunks > 65535) SP_FAIL("rglru: %d chunks are too many for one launch", n_chunks);
    const int col_tiles = (a.size + RG_COLS - 1) / RG_COLS;
    const dim3 grid(parts * col_tiles, n_chunks);
    const bool mma = tensor_cores && g_dt == SP_DT_BF16 && a.size % 8 == 0 && (((uintptr_t)ra | (uintptr_t)ri) & 15) == 0;
    if (mma) {
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
    SP_CHECK_CALL("rglru_scan", sp_launch_dependent(rglru_scan_kernel, dim3((W + 127) / 128, B), dim3(128), 0, stream, a));
    const bool vec = W % 4 == 0 && ld % 4 == 0 && (((uintptr_t)proj | (uintptr_t)av | (uintptr_t)out) & 15) == 0;
    if (vec) SP_CHECK_CALL("rglru_finish", sp_launch_dependent(rglru_finish_kernel<4>, dim3((W + 127) / 128, n_chunks), dim3(256), 0, stream, a));
    else SP_CHECK_CALL("rglru_finish", sp_launch_dependent(rglru_finish_kernel<1>, dim3((W + 31) / 32, n_chunks), dim3(256), 0, stream, a));
    return 0;
}

// A step with one token per sequence.
SP_API int sp_rglru_step(const float* proj, int ld, const float* yb, const float* xb, const float* conv, const float* convb,
                         const void* ra, const void* ri, int g_dt, const float* rab, const float* rib, const float* decay,
                         float* ring, float* state, int n_slots, const int* seq_start, const int* seq_slot, const int* positions,
                         void* out, int out_dt, int B, int W, int taps, int parts, float mult, cudaStream_t stream) {
    if (B <= 0) return 0;
    RgArgs a{proj, ld, yb, xb, conv, convb, ra, ri, g_dt, rab, rib, decay, ring, state, n_slots, seq_start, seq_slot, positions,
             nullptr, nullptr, out, out_dt, B, B, W, taps, parts, parts > 0 ? W / parts : 0, mult};
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
#define RS_LAUNCH(TW, TB) SP_CHECK_CALL("rglru_step", sp_launch_dependent(rglru_step_kernel<TW, TB>, grid, dim3(256), smem, stream, a, row_tiles, vec))
    if (g_dt == SP_DT_BF16) { if (tb == 8) RS_LAUNCH(__nv_bfloat16, 8); else RS_LAUNCH(__nv_bfloat16, 1); }
    else { if (tb == 8) RS_LAUNCH(float, 8); else RS_LAUNCH(float, 1); }
#undef RS_LAUNCH
    return 0;
}
