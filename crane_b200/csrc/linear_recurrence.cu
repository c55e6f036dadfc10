// A gated linear recurrence with a state of one number per channel, behind a short convolution, and what
// surrounds it:
//
//     u = conv(x) + bias                                  (causal, per channel, `taps` taps, no activation)
//     r = sigmoid(R_b u_b + rb),  i = sigmoid(I_b u_b + ib)   (u in equal parts b, a square matrix each)
//     log a = -8 r softplus(lam);   S <- a S + sqrt(1 - a^2) i u;   out = S gelu_tanh(y)
//
// x and y are columns of one merged projection.  `gate_scan_prep` forms, of every token and channel, a and
// b = sqrt(1 - a^2) i u in 32-bit, and of a tile of tokens what its walk comes to: A_t and B_t with S_t = A_t S + B_t for
// the state S before the tile, A_t = 0 from a portion's first token on (the slot's state is in its B_t).  `channel_scan`
// works out the states before the tiles from the tiles' last rows, and the read-outs.  In a step of single tokens the
// first kernel does the walk's one token as well and there is no second one.
// The products with the square matrices: on the bfloat16 path warp-level MMA, u as the sum of two bfloat16 numbers
// (its rounding and what that leaves), so that the gates see u with 16 bits of mantissa; on the 32-bit path, and
// for parts wider than the tensor-core kernel takes, FP32 cores, inner dimension in order.
// The request's slot holds the states [C] and, behind them, the convolution's last inputs as a ring: the input of
// position p lies in row p mod taps of [taps][C].  A single token's input goes to a row that no token of its step
// reads, so the convolution may be read by several CTAs while one of them writes.
#include "common.cuh"

namespace {

constexpr int LIN_MAX_TAPS = 16;
constexpr float LIN_RATE = 8.f;                // log a = -LIN_RATE r softplus(lam)

__device__ __forceinline__ float lin_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }
// On the bfloat16 path: the device's fast forms, errors of a few units in the last place of 32-bit.
__device__ __forceinline__ float lin_sigmoid_fast(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
__device__ __forceinline__ float lin_sqrt_fast(float v) {
    float r;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
__device__ __forceinline__ float lin_gelu_tanh(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// 1 - exp(x) for x <= 0, exp(x) given: near 0 from the series of the exponential, -x (1 + x/2 (1 + x/3 (...))), which
// loses nothing to the subtraction.
__device__ __forceinline__ float one_minus_exp(float x, float exp_x) {
    const float series = -x * fmaf(x * 0.5f, fmaf(x * (1.f / 3.f), fmaf(x * 0.25f, fmaf(x * 0.2f, fmaf(x * (1.f / 6.f), 1.f, 1.f), 1.f), 1.f), 1.f), 1.f);
    return x > -0.25f ? series : 1.f - exp_x;
}

template <typename T>
struct GateScanArgs {
    GemmOut<T> proj;
    int cols, y_off, x_off;                    // row length of the projection; where y and x lie in a row
    const int *tok_entry, *cu_q, *kv_len, *slots;
    int n_slots;
    float* state;                              // [slots][slot_stride]: S at s_off, the ring at ring_off
    long long slot_stride, s_off, ring_off;
    const float *conv_w, *conv_b;              // [taps][C], [C]
    int taps;
    const T* gates;                            // MMA: [2][C][ld] (R's rows, then I's; ld = part width, zero-filled to 16);
                                               // FP32 cores: [2][B][width][width], columns (outputs) side by side
    const float *rb, *ib, *sp;                 // [C]; sp = softplus(lam)
    float* aux;                                // [n][2 C]: A, then B
    T* out;                                    // [n][C] (single tokens)
    int n, C, width, ld;
    int* err;
};

// What a tile needs to know of its tokens.
struct TileToken { int entry, place, start, slot; };     // entry -1: nothing to do

template <typename T>
__device__ __forceinline__ TileToken tile_token(const GateScanArgs<T>& g, int t) {
    TileToken k{-1, 0, 0, 0};
    if (t >= g.n) return k;
    const int e = g.tok_entry[t];
    if (e < 0) return k;
    const int first = g.cu_q[e];
    k.slot = g.slots[e];
    if (k.slot < 0 || k.slot >= g.n_slots) {
        atomicOr(g.err, CRANE_ERR_SLOT_RANGE);
        return k;
    }
    k.entry = e;
    k.place = t - first;                                   // the token's place in its portion
    k.start = g.kv_len[e] - (g.cu_q[e + 1] - first);       // tokens of the request before the step
    return k;
}

// The convolution's input of channel c, `back` tokens before token t.
template <typename T>
__device__ __forceinline__ float conv_input(const GateScanArgs<T>& g, const TileToken& k, int t, int c, int back) {
    if (k.place >= back) return g.proj.load((long long)(t - back) * g.cols + g.x_off + c);
    const int p = k.start + k.place - back;                // before the step: from the ring
    return p >= 0 ? g.state[(long long)k.slot * g.slot_stride + g.ring_off + (long long)(p % g.taps) * g.C + c] : 0.f;
}
template <typename T>
__device__ __forceinline__ float conv_at(const GateScanArgs<T>& g, const TileToken& k, int t, int c) {
    float acc = g.conv_b[c];
    for (int j = 0; j < g.taps; ++j)
        acc = fmaf(g.conv_w[(long long)j * g.C + c], conv_input(g, k, t, c, g.taps - 1 - j), acc);
    return acc;
}

// Channel c: from the two products' sums to the decay and the addend.
template <typename T>
__device__ __forceinline__ void gate_scan_terms(const GateScanArgs<T>& g, int c, float zr, float zi, float u, float& a, float& add) {
    constexpr bool FAST = sizeof(T) == 2;
    zr += g.rb[c];
    zi += g.ib[c];
    const float r = FAST ? lin_sigmoid_fast(zr) : lin_sigmoid(zr), i = FAST ? lin_sigmoid_fast(zi) : lin_sigmoid(zi);
    const float log_a = -LIN_RATE * r * g.sp[c];
    a = expf(log_a);
    const float rest = one_minus_exp(2.f * log_a, a * a);
    add = (FAST ? lin_sqrt_fast(rest) : sqrtf(rest)) * i * u;
}
// A portion's first token: the slot's state joins the addend, and what came before counts no more.
template <typename T>
__device__ __forceinline__ void gate_scan_open(const GateScanArgs<T>& g, const TileToken& k, int c, float& a, float& add) {
    if (k.place != 0) return;
    if (k.start > 0) add = fmaf(g.state[(long long)k.slot * g.slot_stride + g.s_off + c], a, add);
    a = 0.f;
}
// A single token, channel c: the walk, the read-out, the slot.
template <typename T>
__device__ __forceinline__ void gate_scan_single(const GateScanArgs<T>& g, const TileToken& k, int t, int c, float zr, float zi,
                                                 float u) {
    const float x = g.proj.load((long long)t * g.cols + g.x_off + c), y = g.proj.load((long long)t * g.cols + g.y_off + c);
    float* slot = g.state + (long long)k.slot * g.slot_stride;
    float a, add;
    gate_scan_terms(g, c, zr, zi, u, a, add);
    const float s = fmaf(k.start > 0 ? slot[g.s_off + c] : 0.f, a, add);
    slot[g.s_off + c] = s;
    slot[g.ring_off + (long long)(k.start % g.taps) * g.C + c] = x;
    g.out[(long long)t * g.C + c] = from_f32<T>(s * lin_gelu_tanh(y));
}

// ------------------------------------------------------ FP32 cores
// A CTA takes SIMT_TOKENS tokens and 128 columns of one part, a thread per column; u of the whole part in shared
// memory.  Grid (token tiles, parts, column blocks of a part).
constexpr int SIMT_TOKENS = 16;
template <typename T, bool SINGLE>
__global__ void __launch_bounds__(128)
gate_scan_prep_simt_kernel(const GateScanArgs<T> g) {
    extern __shared__ __align__(16) float lin_us[];         // [SIMT_TOKENS][width]
    __shared__ TileToken tok[SIMT_TOKENS];
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * SIMT_TOKENS, part = blockIdx.y;
    if (threadIdx.x < SIMT_TOKENS) tok[threadIdx.x] = tile_token(g, t0 + threadIdx.x);
    __syncthreads();
    for (int x = threadIdx.x; x < SIMT_TOKENS * g.width; x += blockDim.x) {
        const int tt = x / g.width, c = x % g.width;
        lin_us[x] = tok[tt].entry >= 0 ? conv_at(g, tok[tt], t0 + tt, part * g.width + c) : 0.f;
    }
    __syncthreads();
    const int c = blockIdx.z * 128 + threadIdx.x;
    if (c >= g.width) return;
    const T* wr = g.gates + (long long)part * g.width * g.width + c;
    const T* wi = wr + (long long)g.C * g.width;
    float zr[SIMT_TOKENS], zi[SIMT_TOKENS];
#pragma unroll
    for (int tt = 0; tt < SIMT_TOKENS; ++tt) zr[tt] = zi[tt] = 0.f;
    for (int k = 0; k < g.width; ++k) {
        const float a = to_f32(wr[(long long)k * g.width]), b = to_f32(wi[(long long)k * g.width]);
#pragma unroll
        for (int tt = 0; tt < SIMT_TOKENS; ++tt) {
            const float u = lin_us[tt * g.width + k];
            zr[tt] = fmaf(a, u, zr[tt]);
            zi[tt] = fmaf(b, u, zi[tt]);
        }
    }
    const int cc = part * g.width + c;
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int tt = 0; tt < SIMT_TOKENS; ++tt) {
        if (tok[tt].entry < 0) continue;
        if (SINGLE) {
            gate_scan_single(g, tok[tt], t0 + tt, cc, zr[tt], zi[tt], lin_us[tt * g.width + c]);
            continue;
        }
        float a, b;
        gate_scan_terms(g, cc, zr[tt], zi[tt], lin_us[tt * g.width + c], a, b);
        gate_scan_open(g, tok[tt], cc, a, b);
        A *= a;
        B = fmaf(a, B, b);
        float* o = g.aux + (long long)(t0 + tt) * 2 * g.C + cc;
        o[0] = A;
        o[g.C] = B;
    }
}

// ------------------------------------------------------ tensor cores
__device__ __forceinline__ void lin_ldsm_x4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void lin_mma(float (&acc)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(acc[0]), "+f"(acc[1]), "+f"(acc[2]), "+f"(acc[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// u of two neighbouring channels c, c + 1 at token t, everything it reads in flight at once (rows of even length; up to 4
// taps, else one channel after the other).
__device__ __forceinline__ float2 conv_at2(const GateScanArgs<__nv_bfloat16>& g, const TileToken& k, int t, int c) {
    if (g.taps > 4) return make_float2(conv_at(g, k, t, c), conv_at(g, k, t, c + 1));
    float2 x[4], w[4];
    const float2 bias = ld2(g.conv_b + c);
    const float* ring = g.state + (long long)k.slot * g.slot_stride + g.ring_off + c;
#pragma unroll
    for (int back = 0; back < 4; ++back) {
        x[back] = w[back] = make_float2(0.f, 0.f);
        if (back >= g.taps) continue;
        w[back] = ld2(g.conv_w + (long long)(g.taps - 1 - back) * g.C + c);
        const int p = k.start + k.place - back;
        if (k.place >= back) x[back] = g.proj.load2((long long)(t - back) * g.cols + g.x_off + c);
        else if (p >= 0) x[back] = ld2(ring + (long long)(p % g.taps) * g.C);
    }
    float2 u = bias;
#pragma unroll
    for (int back = 3; back >= 0; --back) {
        u.x = fmaf(w[back].x, x[back].x, u.x);
        u.y = fmaf(w[back].y, x[back].y, u.y);
    }
    return u;
}
// u as its rounding and what that leaves.
__device__ __forceinline__ void split_store(__nv_bfloat16* hi, __nv_bfloat16* lo, float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    *(__nv_bfloat162*)hi = h;
    *(__nv_bfloat162*)lo = __floats2bfloat162_rn(a - f.x, b - f.y);
}
// The weights of `cols` columns from c0 on of both matrices: w_s [2][cols][ld + 8].
__device__ __forceinline__ void load_gates(const GateScanArgs<__nv_bfloat16>& g, __nv_bfloat16* w_s, int cols, int base_c, int c0) {
    const int pieces = g.ld >> 3, ldm = g.ld + 8;            // (8 threads a row: a piece each, then the next 8)
    for (int r = threadIdx.x >> 3; r < 2 * cols; r += blockDim.x >> 3) {
        const int m = r >= cols, c = c0 + r - m * cols;
        const __nv_bfloat16* src = g.gates + ((long long)m * g.C + base_c + c) * g.ld;
        for (int q = threadIdx.x & 7; q < pieces; q += 8) {
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (c < g.width) v = *reinterpret_cast<const uint4*>(src + q * 8);
            *reinterpret_cast<uint4*>(w_s + r * ldm + q * 8) = v;
        }
    }
}
// One step of 16 along the inner dimension: 16 tokens (rows from u_hi / u_lo on) by 16 columns of both matrices.
__device__ __forceinline__ void gate_mma_step(float (&zr)[2][4], float (&zi)[2][4], const __nv_bfloat16* u_hi,
                                              const __nv_bfloat16* u_lo, const __nv_bfloat16* wr, const __nv_bfloat16* wi, int ldm,
                                              int ks, int lane) {
    uint32_t ah[4], al[4], b0, b1, b2, b3;
    const int at = (lane & 15) * ldm + ks * 16 + (lane >> 4) * 8;
    const int bt = ((lane & 7) + (lane >> 4) * 8) * ldm + ks * 16 + ((lane >> 3) & 1) * 8;
    lin_ldsm_x4(ah[0], ah[1], ah[2], ah[3], u_hi + at);
    lin_ldsm_x4(al[0], al[1], al[2], al[3], u_lo + at);
    lin_ldsm_x4(b0, b1, b2, b3, wr + bt);
    lin_mma(zr[0], ah, b0, b1);
    lin_mma(zr[1], ah, b2, b3);
    lin_mma(zr[0], al, b0, b1);
    lin_mma(zr[1], al, b2, b3);
    lin_ldsm_x4(b0, b1, b2, b3, wi + bt);
    lin_mma(zi[0], ah, b0, b1);
    lin_mma(zi[1], ah, b2, b3);
    lin_mma(zi[0], al, b0, b1);
    lin_mma(zi[1], al, b2, b3);
}

// Few tokens: a CTA takes 16 tokens and 32 columns of one part, the inner dimension dealt out to FEW_SPLIT pairs of warps
// (16 columns each); the sums meet in shared memory and every thread finishes its share of the tile.  Grid (token tiles,
// parts, column blocks).  Shared memory: u [2][16][ld + 8], both matrices' rows [2][32][ld + 8].
constexpr int FEW_SPLIT = 4, FEW_COLS = 32;
template <bool SINGLE>
__global__ void __launch_bounds__(2 * FEW_SPLIT * 32)
gate_scan_prep_few_kernel(const GateScanArgs<__nv_bfloat16> g, int pairs) {
    extern __shared__ __align__(16) unsigned char lin_smem[];
    __shared__ TileToken tok[16];
    __shared__ float sums[FEW_SPLIT][2][16][FEW_COLS + 1];
    const int ldm = g.ld + 8;
    __nv_bfloat16* u_hi = reinterpret_cast<__nv_bfloat16*>(lin_smem);
    __nv_bfloat16* u_lo = u_hi + 16 * ldm;
    __nv_bfloat16* w_s = u_lo + 16 * ldm;
    const int t0 = blockIdx.x * 16, c0 = blockIdx.z * FEW_COLS, base_c = blockIdx.y * g.width;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_launch_dependents();
    // (the weights depend on no earlier kernel, and what the step's entries are was written before the step began)
    if (threadIdx.x < 16) tok[threadIdx.x] = tile_token(g, t0 + threadIdx.x);
    load_gates(g, w_s, FEW_COLS, base_c, c0);
    __syncthreads();
    pdl_wait();
    const int half = g.ld >> 1;
#pragma unroll 2
    for (int x = threadIdx.x; x < 16 * half; x += blockDim.x) {
        const int tt = x / half, c = 2 * (x % half);
        const TileToken k = tok[tt];
        float2 u = make_float2(0.f, 0.f);
        if (k.entry >= 0) {
            if (pairs && c + 1 < g.width) u = conv_at2(g, k, t0 + tt, base_c + c);
            else {
                if (c < g.width) u.x = conv_at(g, k, t0 + tt, base_c + c);
                if (c + 1 < g.width) u.y = conv_at(g, k, t0 + tt, base_c + c + 1);
            }
        }
        split_store(u_hi + tt * ldm + c, u_lo + tt * ldm + c, u.x, u.y);
    }
    __syncthreads();
    {
        const int wn = warp & 1, wk = warp >> 1;
        float zr[2][4] = {}, zi[2][4] = {};
        for (int ks = wk; ks < (g.ld >> 4); ks += FEW_SPLIT)
            gate_mma_step(zr, zi, u_hi, u_lo, w_s + wn * 16 * ldm, w_s + (FEW_COLS + wn * 16) * ldm, ldm, ks, lane);
#pragma unroll
        for (int b = 0; b < 2; ++b)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int tt = (lane >> 2) + (j >> 1) * 8, c = wn * 16 + b * 8 + 2 * (lane & 3) + (j & 1);
                sums[wk][0][tt][c] = zr[b][j];
                sums[wk][1][tt][c] = zi[b][j];
            }
    }
    __syncthreads();
    for (int x = threadIdx.x; x < 16 * FEW_COLS; x += blockDim.x) {
        const int tt = x / FEW_COLS, cc = x % FEW_COLS, c = c0 + cc;
        if (c >= g.width || tok[tt].entry < 0) continue;
        float zr = 0.f, zi = 0.f;
#pragma unroll
        for (int w = 0; w < FEW_SPLIT; ++w) zr += sums[w][0][tt][cc], zi += sums[w][1][tt][cc];
        const float u = __bfloat162float(u_hi[tt * ldm + c]) + __bfloat162float(u_lo[tt * ldm + c]);
        if (SINGLE) {
            gate_scan_single(g, tok[tt], t0 + tt, base_c + c, zr, zi, u);
            continue;
        }
        float a, b;
        gate_scan_terms(g, base_c + c, zr, zi, u, a, b);
        gate_scan_open(g, tok[tt], base_c + c, a, b);
        sums[0][0][tt][cc] = a;                             // (read by this thread alone)
        sums[0][1][tt][cc] = b;
    }
    if (SINGLE) return;
    __syncthreads();
    if (threadIdx.x < FEW_COLS && c0 + threadIdx.x < g.width) {
        float A = 1.f, B = 0.f;
        for (int tt = 0; tt < 16 && tok[tt].entry >= 0; ++tt) {
            const float a = sums[0][0][tt][threadIdx.x];
            A *= a;
            B = fmaf(a, B, sums[0][1][tt][threadIdx.x]);
            float* o = g.aux + (long long)(t0 + tt) * 2 * g.C + base_c + c0 + threadIdx.x;
            o[0] = A;
            o[g.C] = B;
        }
    }
}

// Many tokens: a CTA takes 48 tokens and wn * 16 columns of one part, 3 x wn warps of 16 tokens and 16 columns.  The
// inputs of the tile's tokens and of the three before it come into shared memory first; a thread then walks a run of
// tokens of two channels with the inputs sliding through registers.  A portion's first tokens, which read the ring, and
// convolutions of more taps go one by one.  Grid (token tiles, parts, column blocks).  Shared memory: inputs
// [51][ld], u [2][48][ld + 8], both matrices' rows [2][wn * 16][ld + 8].
constexpr int MANY_TOKENS = 48, MANY_RUN = 8, MANY_MAX_WN = 5;
// Bytes before the weights: the inputs and u, later the tile's terms in their place.
__host__ __device__ constexpr int many_front(int ld, int cols) {
    const int u = ((MANY_TOKENS + 3) * ld + 2 * MANY_TOKENS * (ld + 8)) * 2, terms = 2 * MANY_TOKENS * (cols + 1) * 4;
    return ((u > terms ? u : terms) + 15) / 16 * 16;
}
__global__ void __launch_bounds__(MANY_TOKENS / 16 * MANY_MAX_WN * 32, 2)
gate_scan_prep_many_kernel(const GateScanArgs<__nv_bfloat16> g, int wn_warps, int pairs, int vec) {
    extern __shared__ __align__(16) unsigned char lin_smem[];
    __shared__ TileToken tok[MANY_TOKENS];
    const int ldm = g.ld + 8, width = g.width, cols = wn_warps * 16;
    __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(lin_smem);
    __nv_bfloat16* u_hi = xs + (MANY_TOKENS + 3) * g.ld;
    __nv_bfloat16* u_lo = u_hi + MANY_TOKENS * ldm;
    __nv_bfloat16* w_s = reinterpret_cast<__nv_bfloat16*>(lin_smem + many_front(g.ld, cols));
    const int t0 = blockIdx.x * MANY_TOKENS, c0 = blockIdx.z * cols, base_c = blockIdx.y * width;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_launch_dependents();
    if (threadIdx.x < MANY_TOKENS) tok[threadIdx.x] = tile_token(g, t0 + threadIdx.x);
    load_gates(g, w_s, cols, base_c, c0);
    pdl_wait();
    if (vec) {                                              // rows of 16-byte pieces
        const int pieces = g.ld >> 3;
        for (int r = threadIdx.x >> 3; r < MANY_TOKENS + 3; r += blockDim.x >> 3) {
            const int t = t0 - 3 + r;
            const __nv_bfloat16* src = g.proj.whole + (long long)t * g.cols + g.x_off + base_c;
            for (int c = (threadIdx.x & 7) * 8; c < pieces * 8; c += 64) {
                uint4 v = make_uint4(0u, 0u, 0u, 0u);
                if (t >= 0 && t < g.n && c < width) v = *reinterpret_cast<const uint4*>(src + c);
                *reinterpret_cast<uint4*>(xs + r * g.ld + c) = v;
            }
        }
    } else {
        const int half = g.ld >> 1;
        for (int x = threadIdx.x; x < (MANY_TOKENS + 3) * half; x += blockDim.x) {
            const int r = x / half, c = x % half * 2, t = t0 - 3 + r;
            float2 v = make_float2(0.f, 0.f);
            if (t >= 0 && t < g.n) {
                const long long at = (long long)t * g.cols + g.x_off + base_c + c;
                if (pairs && c + 1 < width) v = g.proj.load2(at);
                else {
                    if (c < width) v.x = g.proj.load(at);
                    if (c + 1 < width) v.y = g.proj.load(at + 1);
                }
            }
            st2(xs + r * g.ld + c, v.x, v.y);
        }
    }
    __syncthreads();
    {
        const int half = g.ld >> 1;
        for (int x = threadIdx.x; x < half * (MANY_TOKENS / MANY_RUN); x += blockDim.x) {
            const int c = 2 * (x % half), first = x / half * MANY_RUN;
            const bool in0 = c < width, in1 = c + 1 < width;
            float2 w[4], win[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {                   // aligned to the last of 4 taps
                const int tap = j - (4 - g.taps);
                const float* cw = g.conv_w + (long long)tap * g.C + base_c + c;
                w[j] = make_float2(tap >= 0 && in0 ? cw[0] : 0.f, tap >= 0 && in1 ? cw[1] : 0.f);
            }
            const float2 bias = make_float2(in0 ? g.conv_b[base_c + c] : 0.f, in1 ? g.conv_b[base_c + c + 1] : 0.f);
#pragma unroll
            for (int j = 0; j < 3; ++j) win[j] = ld2(xs + (first + j) * g.ld + c);
#pragma unroll
            for (int tt = 0; tt < MANY_RUN; ++tt) {
                const TileToken k = tok[first + tt];
                win[3] = ld2(xs + (first + tt + 3) * g.ld + c);
                float2 u = bias;
#pragma unroll
                for (int j = 0; j < 4; ++j) u.x = fmaf(w[j].x, win[j].x, u.x), u.y = fmaf(w[j].y, win[j].y, u.y);
                if (k.entry < 0) u = make_float2(0.f, 0.f);
                else if (k.place < g.taps - 1 || g.taps > 4)
                    u = make_float2(in0 ? conv_at(g, k, t0 + first + tt, base_c + c) : 0.f,
                                    in1 ? conv_at(g, k, t0 + first + tt, base_c + c + 1) : 0.f);
                split_store(u_hi + (first + tt) * ldm + c, u_lo + (first + tt) * ldm + c, u.x, u.y);
#pragma unroll
                for (int j = 0; j < 3; ++j) win[j] = win[j + 1];
            }
        }
    }
    __syncthreads();
    const int wm = warp % (MANY_TOKENS / 16), wn = warp / (MANY_TOKENS / 16);
    float zr[2][4] = {}, zi[2][4] = {};
    for (int ks = 0; ks < (g.ld >> 4); ++ks)
        gate_mma_step(zr, zi, u_hi + wm * 16 * ldm, u_lo + wm * 16 * ldm, w_s + wn * 16 * ldm, w_s + (cols + wn * 16) * ldm, ldm, ks, lane);
    // the terms of the tile, [48][cols + 1] each, in the place of the inputs and of u
    const int ldt = cols + 1;
    float* ta = reinterpret_cast<float*>(lin_smem);
    float* tb = ta + MANY_TOKENS * ldt;
#pragma unroll
    for (int b = 0; b < 2; ++b)
#pragma unroll
        for (int h = 0; h < 4; ++h) {
            const int tt = wm * 16 + (lane >> 2) + (h >> 1) * 8, c = c0 + wn * 16 + b * 8 + 2 * (lane & 3) + (h & 1);
            float a = 1.f, add = 0.f;                       // (rows of no entry and columns behind the part)
            if (c < width && tok[tt].entry >= 0) {
                const float u = __bfloat162float(u_hi[tt * ldm + c]) + __bfloat162float(u_lo[tt * ldm + c]);
                gate_scan_terms(g, base_c + c, zr[b][h], zi[b][h], u, a, add);
                gate_scan_open(g, tok[tt], base_c + c, a, add);
            }
            zr[b][h] = a;
            zi[b][h] = add;
        }
    __syncthreads();
#pragma unroll
    for (int b = 0; b < 2; ++b)
#pragma unroll
        for (int h = 0; h < 4; ++h) {
            const int tt = wm * 16 + (lane >> 2) + (h >> 1) * 8, cc = wn * 16 + b * 8 + 2 * (lane & 3) + (h & 1);
            ta[tt * ldt + cc] = zr[b][h];
            tb[tt * ldt + cc] = zi[b][h];
        }
    __syncthreads();
    // a thread walks a run of 8 tokens of one column (there are as many runs as threads), the runs meet in shared memory
    {
        const int cc = threadIdx.x % cols, run = threadIdx.x / cols, first = run * MANY_RUN;
        float A = 1.f, B = 0.f;
#pragma unroll
        for (int j = 0; j < MANY_RUN; ++j) {
            const float a = ta[(first + j) * ldt + cc];
            A *= a;
            B = fmaf(a, B, tb[(first + j) * ldt + cc]);
        }
        float2* ends = reinterpret_cast<float2*>(w_s);      // [runs][cols]; the weights have been read
        ends[run * cols + cc] = make_float2(A, B);
        __syncthreads();
        A = 1.f, B = 0.f;
        for (int r = 0; r < run; ++r) {
            const float2 p = ends[r * cols + cc];
            A *= p.x;
            B = fmaf(p.x, B, p.y);
        }
        const int c = c0 + cc;
        float* o = g.aux + (long long)(t0 + first) * 2 * g.C + base_c + c;
#pragma unroll
        for (int j = 0; j < MANY_RUN; ++j, o += 2 * g.C) {
            const float a = ta[(first + j) * ldt + cc];
            A *= a;
            B = fmaf(a, B, tb[(first + j) * ldt + cc]);
            if (c < width && tok[first + j].entry >= 0) {
                o[0] = A;
                o[g.C] = B;
            }
        }
    }
}

// ------------------------------------------------------ the walk
// Grid (tiles of `tile` tokens, the preparation's; blocks of 64 channels); 2 channels a lane, APPLY_ROWS warps that take a
// token each in turn.  The state before the tile is what the tiles before it come to, from the one in which the request
// of the tile's first token began: their last rows, a share of them per warp, put together in shared memory.
constexpr int APPLY_ROWS = 8;
template <typename T>
__global__ void __launch_bounds__(APPLY_ROWS * 32)
channel_scan_kernel(const float* __restrict__ aux, GemmOut<T> proj, int cols, int y_off, int x_off,
                    const int* __restrict__ tok_entry, const int* __restrict__ cu_q, const int* __restrict__ kv_len,
                    const int* __restrict__ slots, int n_slots, float* __restrict__ state, long long slot_stride,
                    long long s_off, long long ring_off, int taps, T* __restrict__ out, int n, int C, int tile, int pairs,
                    int* err) {
    __shared__ float4 part[APPLY_ROWS][32];
    pdl_launch_dependents();
    const int tile_id = blockIdx.x, t0 = tile_id * tile;
    const int e0 = tok_entry[t0];
    if (e0 < 0) return;                                     // nothing but padding from here on
    const int row = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.y * 64 + 2 * lane;
    const bool in0 = c < C, in1 = c + 1 < C;
    const int first_tile = cu_q[e0] / tile;
    pdl_wait();
    auto load = [&](const float* p) {
        if (pairs) return in0 ? ld2(p) : make_float2(0.f, 0.f);
        return make_float2(in0 ? p[0] : 0.f, in1 ? p[1] : 0.f);
    };
    float2 carry = make_float2(0.f, 0.f);
    const int before = tile_id - first_tile;
    if (before > 0) {
        const int per = (before + APPLY_ROWS - 1) / APPLY_ROWS;
        const int lo = first_tile + min(before, row * per), hi = first_tile + min(before, (row + 1) * per);
        float4 s = make_float4(1.f, 1.f, 0.f, 0.f);         // (A, A', B, B')
#pragma unroll 4
        for (int j = lo; j < hi; ++j) {
            const float* p = aux + (long long)((j + 1) * tile - 1) * 2 * C + c;
            const float2 a = load(p), b = load(p + C);
            s = make_float4(s.x * a.x, s.y * a.y, fmaf(a.x, s.z, b.x), fmaf(a.y, s.w, b.y));
        }
        part[row][lane] = s;
        __syncthreads();
#pragma unroll
        for (int r = 0; r < APPLY_ROWS; ++r) {
            const float4 p = part[r][lane];
            carry = make_float2(fmaf(p.x, carry.x, p.z), fmaf(p.y, carry.y, p.w));
        }
    }
    const int end = min(n, t0 + tile);
#pragma unroll 2
    for (int t = t0 + row; t < end; t += APPLY_ROWS) {
        const int e = tok_entry[t];
        if (e < 0) break;
        const int slot = slots[e];
        if (slot < 0 || slot >= n_slots) {
            if (lane == 0) atomicOr(err, CRANE_ERR_SLOT_RANGE);
            continue;
        }
        const float* p = aux + (long long)t * 2 * C + c;
        const float2 a = load(p), b = load(p + C);
        const long long at = (long long)t * cols + c;
        float2 y = make_float2(0.f, 0.f);
        if (pairs) { if (in0) y = proj.load2(at + y_off); }
        else {
            if (in0) y.x = proj.load(at + y_off);
            if (in1) y.y = proj.load(at + y_off + 1);
        }
        const float2 s = make_float2(fmaf(a.x, carry.x, b.x), fmaf(a.y, carry.y, b.y));
        T* o = out + (long long)t * C + c;
        const float ox = s.x * lin_gelu_tanh(y.x), oy = s.y * lin_gelu_tanh(y.y);
        if (pairs) { if (in0) st2(o, ox, oy); }
        else {
            if (in0) o[0] = from_f32<T>(ox);
            if (in1) o[1] = from_f32<T>(oy);
        }
        // a portion's last tokens: the state, and the convolution's last inputs (older ones stay where they are)
        const int back = cu_q[e + 1] - 1 - t;
        if (back < taps) {
            float* mine = state + (long long)slot * slot_stride + c;
            float* ring = mine + ring_off + (long long)((kv_len[e] - 1 - back) % taps) * C;
            if (in0) ring[0] = proj.load(at + x_off);
            if (in1) ring[1] = proj.load(at + x_off + 1);
            if (back == 0) {
                if (in0) mine[s_off] = s.x;
                if (in1) mine[s_off + 1] = s.y;
            }
        }
    }
}

template <typename T, bool SINGLE>
int launch_simt(const GateScanArgs<T>& g, int parts, cudaStream_t st) {
    const size_t smem = (size_t)SIMT_TOKENS * g.width * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const auto kern = gate_scan_prep_simt_kernel<T, SINGLE>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return crane_launch(kern, dim3((g.n + SIMT_TOKENS - 1) / SIMT_TOKENS, parts, (g.width + 127) / 128), dim3(128), smem, st, g);
}

constexpr int LIN_SMEM = 208 * 1024;
int launch_tensor(const GateScanArgs<__nv_bfloat16>& g, int parts, int all_single, cudaStream_t st) {
    static bool configured = false;
    if (!configured) {
        const void* kerns[] = {(const void*)gate_scan_prep_few_kernel<true>, (const void*)gate_scan_prep_few_kernel<false>,
                               (const void*)gate_scan_prep_many_kernel};
        for (const void* k : kerns)
            if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, LIN_SMEM) != cudaSuccess)
                return (int)cudaGetLastError();
        configured = true;
    }
    const int ldm = g.ld + 8;
    // two neighbours a load and a store where every row and every place in it is even
    const int pairs = ((g.C | g.width | g.cols | g.x_off | g.y_off) & 1) == 0 && ((g.slot_stride | g.ring_off | g.proj.part_stride) & 1) == 0 &&
                      (((uintptr_t)g.state | (uintptr_t)g.conv_w | (uintptr_t)g.conv_b) & 7) == 0;
    if (all_single || g.n <= 16) {
        const size_t smem = (size_t)2 * (16 + FEW_COLS) * ldm * sizeof(__nv_bfloat16);
        const auto kern = all_single ? gate_scan_prep_few_kernel<true> : gate_scan_prep_few_kernel<false>;
        return crane_launch(kern, dim3((g.n + 15) / 16, parts, (g.width + FEW_COLS - 1) / FEW_COLS), dim3(2 * FEW_SPLIT * 32), smem,
                            st, g, pairs);
    }
    const int vec = g.proj.parts == nullptr && ((g.width | g.cols | g.x_off) & 7) == 0 && ((uintptr_t)g.proj.whole & 15) == 0;
    const auto smem_for = [&](int w) { return (size_t)many_front(g.ld, w * 16) + (size_t)w * 2 * 16 * ldm * sizeof(__nv_bfloat16); };
    const int groups = (g.width + 15) / 16;
    int wn = groups < MANY_MAX_WN ? groups : MANY_MAX_WN;
    while (wn > 1 && smem_for(wn) > LIN_SMEM) --wn;
    if (smem_for(wn) > LIN_SMEM) return (int)cudaErrorInvalidValue;
    const int blocks = (groups + wn - 1) / wn;
    wn = (groups + blocks - 1) / blocks;                    // (as even as it gets)
    return crane_launch(gate_scan_prep_many_kernel, dim3((g.n + MANY_TOKENS - 1) / MANY_TOKENS, parts, blocks), dim3(MANY_TOKENS / 16 * wn * 32),
                        smem_for(wn), st, g, wn, pairs, vec);
}
int launch_tensor(const GateScanArgs<float>&, int, int, cudaStream_t) { return (int)cudaErrorInvalidValue; }

}  // namespace

// The widest part (rounded up to 16) that the tensor-core kernel takes.
CRANE_API int crane_gate_scan_mma_most() { return 384; }

// `mma` 1: bfloat16 gates [2][C][ld] with ld the part's width rounded up to 16, zero-filled, 16-byte aligned; 0:
// [2][parts][width in][width out].  `all_single`: every entry of the step has one token (or none); `out` [n][C] is
// written and the slots are moved on.  Else `aux` [n][2 C] is written and nothing of the slots.
CRANE_API int crane_gate_scan_prep(int dtype, const void* proj, const float* proj_parts, int n_parts,
                                   long long part_stride, int cols, int y_off, int x_off, const int* tok_entry,
                                   const int* cu_q, const int* kv_len, const int* slots, int n_slots, float* state,
                                   long long slot_stride, long long s_off, long long ring_off, const float* conv_w,
                                   const float* conv_b, int taps, const void* gates, int mma, const float* rb,
                                   const float* ib, const float* sp, float* aux, void* out, int n_tokens, int C,
                                   int parts, int all_single, int* err, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (taps < 1 || taps > LIN_MAX_TAPS || parts <= 0 || C <= 0 || C % parts) return (int)cudaErrorInvalidValue;
    const int width = C / parts, ld = (width + 15) / 16 * 16;
    if (mma && (dtype != 1 || ld > crane_gate_scan_mma_most() || ((uintptr_t)gates & 15))) return (int)cudaErrorInvalidValue;
    DISPATCH_T(dtype, {
        GateScanArgs<T> g{GemmOut<T>{(const T*)proj, proj_parts, n_parts, part_stride}, cols, y_off, x_off, tok_entry, cu_q,
                          kv_len, slots, n_slots, state, slot_stride, s_off, ring_off, conv_w, conv_b, taps, (const T*)gates,
                          rb, ib, sp, aux, (T*)out, n_tokens, C, width, ld, err};
        if (mma) return launch_tensor(g, parts, all_single, st);
        return all_single ? launch_simt<T, true>(g, parts, st) : launch_simt<T, false>(g, parts, st);
    });
}

// The tokens of a tile of `crane_gate_scan_prep` for these arguments (not in a step of single tokens).
CRANE_API int crane_gate_scan_tile(int mma, int n_tokens) { return !mma || n_tokens <= 16 ? 16 : MANY_TOKENS; }

CRANE_API int crane_channel_scan(int dtype, const float* aux, const void* proj, const float* proj_parts, int n_parts,
                                 long long part_stride, int cols, int y_off, int x_off, const int* tok_entry,
                                 const int* cu_q, const int* kv_len, const int* slots, int n_slots, float* state,
                                 long long slot_stride, long long s_off, long long ring_off, int taps, void* out,
                                 int n_tokens, int C, int mma, int* err, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (taps < 1 || taps > LIN_MAX_TAPS || C <= 0) return (int)cudaErrorInvalidValue;
    const int tile = crane_gate_scan_tile(mma, n_tokens);
    const int pairs = ((C | cols | y_off) & 1) == 0 && (part_stride & 1) == 0 && ((uintptr_t)aux & 7) == 0;
    DISPATCH_T(dtype, {
        GemmOut<T> p{(const T*)proj, proj_parts, n_parts, part_stride};
        return crane_launch(channel_scan_kernel<T>, dim3((n_tokens + tile - 1) / tile, (C + 63) / 64), dim3(APPLY_ROWS * 32), 0, st,
                            aux, p, cols, y_off, x_off, tok_entry, cu_q, kv_len, slots, n_slots, state, slot_stride, s_off,
                            ring_off, taps, (T*)out, n_tokens, C, tile, pairs, err);
    });
}
