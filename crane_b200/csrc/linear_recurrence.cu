// A gated linear recurrence with a state of one number per channel, behind a short convolution, and what
// surrounds it:
//
//     u = conv(x) + bias                                  (causal, per channel, `taps` taps, no activation)
//     r = sigmoid(R_b u_b + rb),  i = sigmoid(I_b u_b + ib)   (u in equal parts b, a square matrix each)
//     log a = -8 r softplus(lam);   S <- a S + sqrt(1 - a^2) i u;   out = S gelu_tanh(y)
//
// x and y are columns of one merged projection.  `gate_scan_prep` forms, of every token and channel, a and
// sqrt(1 - a^2) i u in 32-bit; `channel_scan` walks each request's tokens.  In a step of single tokens the first
// kernel does the walk's one token as well and there is no second one.
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
__device__ __forceinline__ float lin_gelu_tanh(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
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
    float* aux;                                // [n][2 C]: a, then the addend
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

// Token t, channel c: from the two products' sums to what the walk needs, or, SINGLE, through the walk.
template <typename T, bool SINGLE>
__device__ __forceinline__ void gate_scan_finish(const GateScanArgs<T>& g, const TileToken& k, int t, int c, float zr,
                                                 float zi, float u) {
    const float r = lin_sigmoid(zr + g.rb[c]), i = lin_sigmoid(zi + g.ib[c]);
    const float log_a = -LIN_RATE * r * g.sp[c];
    const float a = expf(log_a), add = sqrtf(-expm1f(2.f * log_a)) * i * u;
    if (!SINGLE) {
        float* o = g.aux + (long long)t * 2 * g.C;
        o[c] = a;
        o[g.C + c] = add;
        return;
    }
    float* slot = g.state + (long long)k.slot * g.slot_stride;
    const float s = fmaf(k.start > 0 ? slot[g.s_off + c] : 0.f, a, add);
    slot[g.s_off + c] = s;
    slot[g.ring_off + (long long)(k.start % g.taps) * g.C + c] = g.proj.load((long long)t * g.cols + g.x_off + c);
    g.out[(long long)t * g.C + c] = from_f32<T>(s * lin_gelu_tanh(g.proj.load((long long)t * g.cols + g.y_off + c)));
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
#pragma unroll
    for (int tt = 0; tt < SIMT_TOKENS; ++tt)
        if (tok[tt].entry >= 0)
            gate_scan_finish<T, SINGLE>(g, tok[tt], t0 + tt, part * g.width + c, zr[tt], zi[tt], lin_us[tt * g.width + c]);
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

// TOKENS x COLS of one part by TOKENS / 16 x (COLS / 16 / KSPLIT...) warps: WM x WN x WK warps, a warp 16 tokens and
// COLS / WN columns (of both products) over every WK-th step of 16 along the inner dimension; with WK = 2 the second
// half's sums go through shared memory.  Grid (token tiles, parts, column blocks of a part).
// Shared memory: u's two parts [2][TOKENS][ld + 8], both matrices' rows [2][COLS][ld + 8], bfloat16.
template <int TOKENS, int COLS, int WN, int WK, bool SINGLE>
__global__ void __launch_bounds__(TOKENS / 16 * WN * WK * 32)
gate_scan_prep_mma_kernel(const GateScanArgs<__nv_bfloat16> g) {
    constexpr int WM = TOKENS / 16, NT = WM * WN * WK * 32;
    constexpr int NB = COLS / WN / 8;                       // blocks of 8 columns a warp takes
    static_assert(NB == 1 || NB % 2 == 0, "one block of 8 columns, or pairs of them");
    extern __shared__ __align__(16) unsigned char lin_smem[];
    __shared__ TileToken tok[TOKENS];
    const int ldm = g.ld + 8;
    __nv_bfloat16* u_hi = reinterpret_cast<__nv_bfloat16*>(lin_smem);
    __nv_bfloat16* u_lo = u_hi + TOKENS * ldm;
    __nv_bfloat16* w_s = u_lo + TOKENS * ldm;
    const int t0 = blockIdx.x * TOKENS, part = blockIdx.y, c0 = blockIdx.z * COLS;
    const int width = g.width, base_c = part * width;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad = lane >> 2, t4 = lane & 3;
    pdl_launch_dependents();
    // the weights depend on no earlier kernel
    const int pieces = g.ld >> 3;
    for (int x = threadIdx.x; x < 2 * COLS * pieces; x += NT) {
        const int r = x / pieces, q = x % pieces, m = r / COLS, c = c0 + r % COLS;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (c < width) v = *reinterpret_cast<const uint4*>(g.gates + ((long long)m * g.C + base_c + c) * g.ld + q * 8);
        *reinterpret_cast<uint4*>(w_s + r * ldm + q * 8) = v;
    }
    pdl_wait();
    if (threadIdx.x < TOKENS) tok[threadIdx.x] = tile_token(g, t0 + threadIdx.x);
    __syncthreads();
    // u of the part: a thread walks a run of tokens of one channel with the inputs sliding through registers
    // (up to 4 taps), so that each is fetched once
    constexpr int RUN = TOKENS >= 64 ? 16 : TOKENS >= 32 ? 8 : 1;
    for (int x = threadIdx.x; x < g.ld * (TOKENS / RUN); x += NT) {
        const int c = x % g.ld, first = x / g.ld * RUN;
        if (c >= width || (RUN == 1 && tok[first].entry < 0)) {
#pragma unroll
            for (int tt = 0; tt < RUN; ++tt)
                u_hi[(first + tt) * ldm + c] = u_lo[(first + tt) * ldm + c] = __float2bfloat16_rn(0.f);
            continue;
        }
        const int cc = base_c + c;
        float wv[4], win[4];
        const bool slide = RUN > 1 && g.taps <= 4;
        if (slide) {
#pragma unroll
            for (int j = 0; j < 4; ++j) {                   // aligned to the last of 4 taps
                wv[j] = j >= 4 - g.taps ? g.conv_w[(long long)(j - (4 - g.taps)) * g.C + cc] : 0.f;
                win[j] = 0.f;
            }
        }
        const float bias = g.conv_b[cc];
#pragma unroll
        for (int tt = 0; tt < RUN; ++tt) {
            const TileToken k = tok[first + tt];
            float u = 0.f;
            if (k.entry >= 0) {
                if (slide) {
                    const int t = t0 + first + tt;
                    if (tt == 0 || k.place == 0) {          // a run's or a portion's beginning: the inputs before it
#pragma unroll
                        for (int j = 0; j < 3; ++j) win[j] = 3 - j < g.taps ? conv_input(g, k, t, cc, 3 - j) : 0.f;
                    }
                    win[3] = g.proj.load((long long)t * g.cols + g.x_off + cc);
                    u = bias;
#pragma unroll
                    for (int j = 0; j < 4; ++j) u = fmaf(wv[j], win[j], u);
#pragma unroll
                    for (int j = 0; j < 3; ++j) win[j] = win[j + 1];
                } else {
                    u = conv_at(g, k, t0 + first + tt, cc);
                }
            }
            const __nv_bfloat16 hi = __float2bfloat16_rn(u);
            u_hi[(first + tt) * ldm + c] = hi;
            u_lo[(first + tt) * ldm + c] = __float2bfloat16_rn(u - __bfloat162float(hi));
        }
    }
    __syncthreads();
    const int wm = warp % WM, wn = warp / WM % WN, wk = warp / (WM * WN);
    float zr[NB][4], zi[NB][4];
#pragma unroll
    for (int b = 0; b < NB; ++b) zr[b][0] = zr[b][1] = zr[b][2] = zr[b][3] = zi[b][0] = zi[b][1] = zi[b][2] = zi[b][3] = 0.f;
    const int wcol = wn * NB * 8;
    for (int ks = wk; ks < (g.ld >> 4); ks += WK) {
        uint32_t ah[4], al[4];
        const int at = (wm * 16 + (lane & 15)) * ldm + ks * 16 + (lane >> 4) * 8;
        lin_ldsm_x4(ah[0], ah[1], ah[2], ah[3], u_hi + at);
        lin_ldsm_x4(al[0], al[1], al[2], al[3], u_lo + at);
        if (NB == 1) {
            // one load brings the 8 columns of both matrices: lanes 0..15 R's two halves of 8, lanes 16..31 I's
            uint32_t b0, b1, b2, b3;
            lin_ldsm_x4(b0, b1, b2, b3, w_s + ((lane >> 4) * COLS + wcol + (lane & 7)) * ldm + ks * 16 + ((lane >> 3) & 1) * 8);
            lin_mma(zr[0], ah, b0, b1);
            lin_mma(zi[0], ah, b2, b3);
            lin_mma(zr[0], al, b0, b1);
            lin_mma(zi[0], al, b2, b3);
        } else {
#pragma unroll
            for (int b = 0; b + 1 < NB; b += 2) {
                const int row = wcol + b * 8 + (lane & 7) + (lane >> 4) * 8, col = ks * 16 + ((lane >> 3) & 1) * 8;
                uint32_t b0, b1, b2, b3;
                lin_ldsm_x4(b0, b1, b2, b3, w_s + row * ldm + col);
                lin_mma(zr[b], ah, b0, b1);
                lin_mma(zr[b + 1], ah, b2, b3);
                lin_mma(zr[b], al, b0, b1);
                lin_mma(zr[b + 1], al, b2, b3);
                lin_ldsm_x4(b0, b1, b2, b3, w_s + (COLS + row) * ldm + col);
                lin_mma(zi[b], ah, b0, b1);
                lin_mma(zi[b + 1], ah, b2, b3);
                lin_mma(zi[b], al, b0, b1);
                lin_mma(zi[b + 1], al, b2, b3);
            }
        }
    }
    if (WK == 2) {
        __shared__ float half[WK == 2 ? WM * WN * 32 : 1][NB * 8 + 1];
        float* mine = half[(wn * WM + wm) * 32 + lane];
        if (wk == 1) {
#pragma unroll
            for (int b = 0; b < NB; ++b)
#pragma unroll
                for (int j = 0; j < 4; ++j) mine[b * 8 + j] = zr[b][j], mine[b * 8 + 4 + j] = zi[b][j];
        }
        __syncthreads();
        if (wk == 1) return;
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int j = 0; j < 4; ++j) zr[b][j] += mine[b * 8 + j], zi[b][j] += mine[b * 8 + 4 + j];
    }
#pragma unroll
    for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int tt = wm * 16 + quad + (j >> 1) * 8, c = c0 + wcol + b * 8 + 2 * t4 + (j & 1);
            if (c >= width || tok[tt].entry < 0) continue;
            const float u = __bfloat162float(u_hi[tt * ldm + c]) + __bfloat162float(u_lo[tt * ldm + c]);
            gate_scan_finish<__nv_bfloat16, SINGLE>(g, tok[tt], t0 + tt, base_c + c, zr[b][j], zi[b][j], u);
        }
}

// ------------------------------------------------------ the walk
// Grid (blocks of 32 channels, entries); a lane per channel, a warp per run of RUN tokens of a round of WARPS * RUN.
// A run is first composed to (product of the a's, its sum from zero); from the runs' pairs every warp works out the
// state before its run, and walks it.  The last warp's state begins the next round.
constexpr int SCAN_WARPS = 16, SCAN_RUN = 8;
template <typename T>
__global__ void __launch_bounds__(SCAN_WARPS * 32)
channel_scan_kernel(const float* __restrict__ aux, GemmOut<T> proj, int cols, int y_off, int x_off,
                    const int* __restrict__ cu_q, const int* __restrict__ kv_len, const int* __restrict__ slots,
                    int n_slots, float* __restrict__ state, long long slot_stride, long long s_off, long long ring_off,
                    int taps, T* __restrict__ out, int C, int* err) {
    __shared__ float2 pair[2][SCAN_WARPS][32];
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.y;
    const int first = cu_q[e], q_len = cu_q[e + 1] - first;
    if (q_len <= 0) return;                                 // an entry that pads the step: no slot is touched
    const int slot = slots[e];
    if (slot < 0 || slot >= n_slots) {
        if (threadIdx.x == 0) atomicOr(err, CRANE_ERR_SLOT_RANGE);
        return;
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * 32 + lane;
    const bool live = c < C;
    const int start = kv_len[e] - q_len;
    float* mine = state + (long long)slot * slot_stride;
    float s0 = live && start > 0 ? mine[s_off + c] : 0.f;    // the state before the round
    constexpr int ROUND = SCAN_WARPS * SCAN_RUN;
    float a[SCAN_RUN], b[SCAN_RUN], an[SCAN_RUN], bn[SCAN_RUN];
    auto fetch = [&](int t, float (&pa)[SCAN_RUN], float (&pb)[SCAN_RUN]) {       // tokens past the end change nothing
#pragma unroll
        for (int j = 0; j < SCAN_RUN; ++j) {
            const bool in = live && t + j < q_len;
            const float* row = aux + (long long)(first + t + j) * 2 * C + c;
            pa[j] = in ? row[0] : 1.f;
            pb[j] = in ? row[C] : 0.f;
        }
    };
    fetch(warp * SCAN_RUN, a, b);
    for (int t0 = 0, it = 0; t0 < q_len; t0 += ROUND, ++it) {
        const int t = t0 + warp * SCAN_RUN;
        if (t0 + ROUND < q_len) fetch(t + ROUND, an, bn);
        float y[SCAN_RUN];
#pragma unroll
        for (int j = 0; j < SCAN_RUN; ++j)
            y[j] = live && t + j < q_len ? proj.load((long long)(first + t + j) * cols + y_off + c) : 0.f;
        float A = 1.f, B = 0.f;
#pragma unroll
        for (int j = 0; j < SCAN_RUN; ++j) {
            B = fmaf(a[j], B, b[j]);
            A *= a[j];
        }
        pair[it & 1][warp][lane] = make_float2(A, B);
        __syncthreads();
        float s = s0, mine_s = s0;
#pragma unroll
        for (int w = 0; w < SCAN_WARPS; ++w) {
            if (w == warp) mine_s = s;
            const float2 p = pair[it & 1][w][lane];
            s = fmaf(p.x, s, p.y);
        }
        s0 = s;
#pragma unroll
        for (int j = 0; j < SCAN_RUN; ++j) {
            mine_s = fmaf(a[j], mine_s, b[j]);
            if (live && t + j < q_len)
                out[(long long)(first + t + j) * C + c] = from_f32<T>(mine_s * lin_gelu_tanh(y[j]));
            a[j] = an[j];
            b[j] = bn[j];
        }
    }
    if (!live) return;
    if (warp == 0) mine[s_off + c] = s0;
    // the last inputs of the convolution: those of this step (older ones stay where they are)
    for (int back = warp; back < taps && back < q_len; back += SCAN_WARPS) {
        const int p = kv_len[e] - 1 - back;
        mine[ring_off + (long long)(p % taps) * C + c] = proj.load((long long)(first + q_len - 1 - back) * cols + x_off + c);
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

template <int TOKENS, int COLS, int WN, int WK, bool SINGLE>
int launch_mma(const GateScanArgs<__nv_bfloat16>& g, int parts, cudaStream_t st) {
    const size_t smem = (size_t)2 * (TOKENS + COLS) * (g.ld + 8) * sizeof(__nv_bfloat16);
    const auto kern = gate_scan_prep_mma_kernel<TOKENS, COLS, WN, WK, SINGLE>;
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 208 * 1024) != cudaSuccess)
            return (int)cudaGetLastError();
        configured = true;
    }
    if (smem > 208 * 1024) return (int)cudaErrorInvalidValue;
    return crane_launch(kern, dim3((g.n + TOKENS - 1) / TOKENS, parts, (g.width + COLS - 1) / COLS),
                        dim3(TOKENS / 16 * WN * WK * 32), smem, st, g);
}

int launch_tensor(const GateScanArgs<__nv_bfloat16>& g, int parts, int all_single, cudaStream_t st) {
    if (all_single) return g.n <= 16 ? launch_mma<16, 16, 2, 2, true>(g, parts, st) : launch_mma<32, 32, 2, 1, true>(g, parts, st);
    return g.n <= 16 ? launch_mma<16, 16, 2, 2, false>(g, parts, st) : launch_mma<64, 64, 2, 1, false>(g, parts, st);
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

CRANE_API int crane_channel_scan(int dtype, const float* aux, const void* proj, const float* proj_parts, int n_parts,
                                 long long part_stride, int cols, int y_off, int x_off, const int* cu_q,
                                 const int* kv_len, const int* slots, int n_slots, float* state, long long slot_stride,
                                 long long s_off, long long ring_off, int taps, void* out, int n_entries, int C,
                                 int* err, cudaStream_t st) {
    if (n_entries <= 0) return 0;
    if (taps < 1 || taps > LIN_MAX_TAPS || C <= 0) return (int)cudaErrorInvalidValue;
    DISPATCH_T(dtype, {
        GemmOut<T> p{(const T*)proj, proj_parts, n_parts, part_stride};
        return crane_launch(channel_scan_kernel<T>, dim3((C + 31) / 32, n_entries), dim3(SCAN_WARPS * 32), 0, st, aux, p,
                            cols, y_off, x_off, cu_q, kv_len, slots, n_slots, state, slot_stride, s_off, ring_off, taps,
                            (T*)out, C, err);
    });
}
