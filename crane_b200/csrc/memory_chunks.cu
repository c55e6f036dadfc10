// The matrix memory with exponential gates of `recurrent_parts.cu` (scan mode `gated`) for portions of many tokens, in
// chunks of 64 tokens on the tensor cores.  With log w_t and log b_t (both <= 0) from `exp_gate_prep` and
// L_t = sum of log w over the chunk's tokens up to t, a chunk that begins with state S gives
//
//     o_t = exp(L_t) S^T q_t + sum over s <= t of  exp(L_t - L_s + log b_s) (q_t . k_s) v_s
//     S  <- exp(L_63) S + sum over s of  exp(L_63 - L_s + log b_s) k_s v_s^T
//
// No exponent is above 0.  The normaliser is column dv of S, whose values are 1.  A CTA has one (request, head) and 16
// columns; it walks the request's chunks with S in 32-bit accumulators.  Products are warp-level MMA with 32-bit sums;
// q, k and v are bfloat16 as the projection left them, and what is 32-bit (S, the weighted scores, the weighted values)
// enters a product as the sum of two bfloat16 numbers, its rounding and what that leaves.
// Grid (blocks of 16 columns of dv + 1, heads, entries); entries of fewer than `min_len` tokens are another kernel's.
#include "common.cuh"

namespace {

constexpr int CHUNK = 64, CB = 16, LDV = CB + 8, LDP = CHUNK + 8;

__device__ __forceinline__ uint32_t mc_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mc_ldsm(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mc_smem(p)));
}
__device__ __forceinline__ void mc_ldsm_t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mc_smem(p)));
}
__device__ __forceinline__ void mc_mma(float (&acc)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(acc[0]), "+f"(acc[1]), "+f"(acc[2]), "+f"(acc[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mc_copy16(void* dst, const void* src, bool in) {       // zeros where `in` is false
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mc_smem(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void mc_copy4(void* dst, const void* src, bool in) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(mc_smem(dst)), "l"(src), "r"(in ? 4 : 0) : "memory");
}
__device__ __forceinline__ void mc_split(__nv_bfloat16* hi, __nv_bfloat16* lo, float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    *(__nv_bfloat162*)hi = h;
    *(__nv_bfloat162*)lo = __floats2bfloat162_rn(a - f.x, b - f.y);
}

// TILES: row tiles of 16 of the state a warp holds (keys of up to 128 TILES elements).
template <int TILES>
__global__ void __launch_bounds__(256)
memory_chunks_kernel(const __nv_bfloat16* __restrict__ proj, int cols, int q_off, int k_off, int v_off,
                     const float* __restrict__ logs, int logs_ld, const int* __restrict__ cu_q,
                     const int* __restrict__ kv_len, const int* __restrict__ slots, int n_slots, float* __restrict__ state,
                     long long slot_stride, float* __restrict__ o_raw, float* __restrict__ den, int H, int d, int dv,
                     int rows_per_lane, int lanes, float q_scale, int min_len, int* err) {
    extern __shared__ __align__(16) unsigned char mc_raw[];
    const int ldk = d + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(mc_raw);         // [2][64][ldk]
    __nv_bfloat16* ks = qs + 2 * CHUNK * ldk;                              // [2][64][ldk]
    __nv_bfloat16* vs = ks + 2 * CHUNK * ldk;                              // [2][64][LDV]
    __nv_bfloat16* wv_hi = vs + 2 * CHUNK * LDV;                           // [64][LDV]  weighted values
    __nv_bfloat16* wv_lo = wv_hi + CHUNK * LDV;
    __nv_bfloat16* p_hi = wv_lo + CHUNK * LDV;                             // [64][LDP]  weighted scores
    __nv_bfloat16* p_lo = p_hi + CHUNK * LDP;
    __nv_bfloat16* s_hi = p_lo + CHUNK * LDP;                              // [d][LDV]
    __nv_bfloat16* s_lo = s_hi + d * LDV;
    float* lw = reinterpret_cast<float*>(s_lo + d * LDV);                  // [2][64]
    float* lb = lw + 2 * CHUNK;                                            // [2][64]
    float* sum = lb + 2 * CHUNK;                                           // [8 warps][64]  L
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * CB;
    const int first = cu_q[e], q_len = cu_q[e + 1] - first;
    if (q_len < min_len) return;
    const int slot = slots[e];
    if (slot < 0 || slot >= n_slots) {
        if (threadIdx.x == 0) atomicOr(err, CRANE_ERR_SLOT_RANGE);
        return;
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad = lane >> 2, t4 = lane & 3;
    const int dvt = dv + 1;
    const int k_pieces = d >> 3;
    auto fetch = [&](int t0, int buf) {
        const int nt = q_len - t0;
        for (int x = threadIdx.x; x < CHUNK * k_pieces; x += 256) {
            const int tt = x / k_pieces, p = (x % k_pieces) * 8;
            const bool in = tt < nt;
            const __nv_bfloat16* row = proj + (long long)(first + t0 + (in ? tt : 0)) * cols + h * d + p;
            mc_copy16(qs + (buf * CHUNK + tt) * ldk + p, row + q_off, in);
            mc_copy16(ks + (buf * CHUNK + tt) * ldk + p, row + k_off, in);
        }
        if (threadIdx.x < 2 * CHUNK) {
            const int tt = threadIdx.x >> 1, p = (threadIdx.x & 1) * 8;
            const bool in = tt < nt;
            if (c0 + p < dv)
                mc_copy16(vs + (buf * CHUNK + tt) * LDV + p, proj + (long long)(first + t0 + (in ? tt : 0)) * cols + v_off + h * dv + c0 + p, in);
        } else {
            const int tt = (threadIdx.x - 2 * CHUNK) & (CHUNK - 1), which = (threadIdx.x - 2 * CHUNK) >> 6;
            const bool in = tt < nt;
            mc_copy4((which ? lb : lw) + buf * CHUNK + tt, logs + (long long)(first + t0 + (in ? tt : 0)) * logs_ld + which * H + h, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // the columns behind dv: the normaliser's values are 1, what is behind it is 0
    for (int x = threadIdx.x; x < 2 * CHUNK * CB; x += 256) {
        const int c = c0 + x % CB;
        if (c >= dv) vs[x / CB * LDV + x % CB] = __float2bfloat16_rn(c == dv ? 1.f : 0.f);
    }
    fetch(0, 0);
    // the state: a warp's tiles of 16 rows x 16 columns
    float s[TILES][2][4];
    float* sp = state + (long long)slot * slot_stride + (long long)h * rows_per_lane * dvt * lanes;
    auto place = [&](int r, int c) { return ((long long)(r % rows_per_lane) * dvt + c) * lanes + r / rows_per_lane; };
    const bool fresh = kv_len[e] == q_len;
    auto keep_split = [&]() {
#pragma unroll
        for (int i = 0; i < TILES; ++i) {
            const int r = (warp * TILES + i) * 16 + quad;
            if (r >= d) continue;
#pragma unroll
            for (int b = 0; b < 2; ++b)
#pragma unroll
                for (int hh = 0; hh < 2; ++hh) {
                    const int at = (r + 8 * hh) * LDV + b * 8 + 2 * t4;
                    mc_split(s_hi + at, s_lo + at, s[i][b][2 * hh], s[i][b][2 * hh + 1]);
                }
        }
    };
#pragma unroll
    for (int i = 0; i < TILES; ++i)
#pragma unroll
        for (int b = 0; b < 2; ++b)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int r = (warp * TILES + i) * 16 + quad + (j >> 1) * 8, c = c0 + b * 8 + 2 * t4 + (j & 1);
                s[i][b][j] = (!fresh && r < d && c < dvt) ? sp[place(r, c)] : 0.f;
            }
    keep_split();
    const int rt = warp & 3, half = warp >> 2;               // 16 rows (tokens); 32 keys, or 8 columns
    float* my_sum = sum + warp * CHUNK;
    for (int t0 = 0, it = 0; t0 < q_len; t0 += CHUNK, ++it) {
        const int buf = it & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                     // the chunk is there; the one before has been read out
        if (t0 + CHUNK < q_len) fetch(t0 + CHUNK, buf ^ 1);
        const __nv_bfloat16 *q = qs + buf * CHUNK * ldk, *k = ks + buf * CHUNK * ldk, *v = vs + buf * CHUNK * LDV;
        {                                                    // L, every warp for itself: two tokens a lane
            const float2 w = ld2(lw + buf * CHUNK + 2 * lane);
            float run = w.x + w.y;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float p = __shfl_up_sync(0xffffffffu, run, o);
                if (lane >= o) run += p;
            }
            st2(my_sum + 2 * lane, run - w.y, run);
            __syncwarp();
        }
        const float* lbp = lb + buf * CHUNK;
        const float l_end = my_sum[CHUNK - 1];
        // weighted values: 64 x 16, four elements a thread
        {
            const int tt = threadIdx.x >> 2, c = (threadIdx.x & 3) * 4;
            const float f = expf(l_end - my_sum[tt] + lbp[tt]);
            const float2 a = ld2(v + tt * LDV + c), b = ld2(v + tt * LDV + c + 2);
            mc_split(wv_hi + tt * LDV + c, wv_lo + tt * LDV + c, a.x * f, a.y * f);
            mc_split(wv_hi + tt * LDV + c + 2, wv_lo + tt * LDV + c + 2, b.x * f, b.y * f);
        }
        // scores of 16 tokens x 32 keys (none where all keys come later), and the state's part of 16 tokens x 8 columns
        float sc[4][4] = {}, o[4] = {};
        const bool scores = half * 32 <= rt * 16 + 15;
        for (int kk = 0; kk < (d >> 4); ++kk) {
            uint32_t a[4], b[4];
            mc_ldsm(a, q + (rt * 16 + (lane & 15)) * ldk + kk * 16 + (lane >> 4) * 8);
            mc_ldsm_t(b, (lane < 16 ? s_hi : s_lo) + (kk * 16 + (lane & 15)) * LDV + half * 8);
            mc_mma(o, a, b[0], b[1]);
            mc_mma(o, a, b[2], b[3]);
            if (scores) {
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    mc_ldsm(b, k + (half * 32 + j * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + kk * 16 + ((lane >> 3) & 1) * 8);
                    mc_mma(sc[2 * j], a, b[0], b[1]);
                    mc_mma(sc[2 * j + 1], a, b[2], b[3]);
                }
            }
        }
        const int ta = rt * 16 + quad;
        const float la = my_sum[ta], lc = my_sum[ta + 8];
        if (scores) {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int key = half * 32 + j * 8 + 2 * t4;
                const float2 ls = ld2(my_sum + key), bs = ld2(lbp + key);
                const float g0 = bs.x - ls.x, g1 = bs.y - ls.y;
                const float a0 = key <= ta ? sc[j][0] * q_scale * expf(la + g0) : 0.f;
                const float a1 = key + 1 <= ta ? sc[j][1] * q_scale * expf(la + g1) : 0.f;
                const float a2 = key <= ta + 8 ? sc[j][2] * q_scale * expf(lc + g0) : 0.f;
                const float a3 = key + 1 <= ta + 8 ? sc[j][3] * q_scale * expf(lc + g1) : 0.f;
                mc_split(p_hi + ta * LDP + key, p_lo + ta * LDP + key, a0, a1);
                mc_split(p_hi + (ta + 8) * LDP + key, p_lo + (ta + 8) * LDP + key, a2, a3);
            }
        }
        __syncthreads();                                     // weighted scores and values are there; the state has been read
        {
            const float fa = expf(la) * q_scale, fc = expf(lc) * q_scale;
            o[0] *= fa, o[1] *= fa, o[2] *= fc, o[3] *= fc;
            for (int kk = 0; kk <= rt; ++kk) {               // (later keys weigh nothing)
                uint32_t ah[4], al[4], b[4];
                mc_ldsm(ah, p_hi + (rt * 16 + (lane & 15)) * LDP + kk * 16 + (lane >> 4) * 8);
                mc_ldsm(al, p_lo + (rt * 16 + (lane & 15)) * LDP + kk * 16 + (lane >> 4) * 8);
                mc_ldsm_t(b, v + (kk * 16 + (lane & 15)) * LDV + (lane >> 4) * 8);
                mc_mma(o, ah, half ? b[2] : b[0], half ? b[3] : b[1]);
                mc_mma(o, al, half ? b[2] : b[0], half ? b[3] : b[1]);
            }
            const int c = c0 + half * 8 + 2 * t4;
#pragma unroll
            for (int hh = 0; hh < 2; ++hh) {
                const int tt = ta + 8 * hh;
                if (t0 + tt >= q_len) continue;
                const long long row = first + t0 + tt;
                if (c < dv) st2(o_raw + row * H * dv + h * dv + c, o[2 * hh], o[2 * hh + 1]);
                else if (c == dv) den[row * H + h] = o[2 * hh];
            }
        }
        const float keep = expf(l_end);
#pragma unroll
        for (int i = 0; i < TILES; ++i) {
            const int r0 = (warp * TILES + i) * 16;
            if (r0 >= d) continue;
#pragma unroll
            for (int b = 0; b < 2; ++b)
#pragma unroll
                for (int j = 0; j < 4; ++j) s[i][b][j] *= keep;
#pragma unroll
            for (int kk = 0; kk < CHUNK / 16; ++kk) {
                uint32_t a[4], bh[4], bl[4];
                mc_ldsm_t(a, k + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + r0 + ((lane >> 3) & 1) * 8);
                mc_ldsm_t(bh, wv_hi + (kk * 16 + (lane & 15)) * LDV + (lane >> 4) * 8);
                mc_ldsm_t(bl, wv_lo + (kk * 16 + (lane & 15)) * LDV + (lane >> 4) * 8);
                mc_mma(s[i][0], a, bh[0], bh[1]);
                mc_mma(s[i][1], a, bh[2], bh[3]);
                mc_mma(s[i][0], a, bl[0], bl[1]);
                mc_mma(s[i][1], a, bl[2], bl[3]);
            }
        }
        keep_split();
    }
#pragma unroll
    for (int i = 0; i < TILES; ++i)
#pragma unroll
        for (int b = 0; b < 2; ++b)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int r = (warp * TILES + i) * 16 + quad + (j >> 1) * 8, c = c0 + b * 8 + 2 * t4 + (j & 1);
                if (r < d && c < dvt) sp[place(r, c)] = s[i][b][j];
            }
}

size_t memory_chunks_smem(int d) {
    const size_t ldk = d + 8;
    return (4 * CHUNK * ldk + 4 * CHUNK * LDV + 2 * CHUNK * LDP + 2 * (size_t)d * LDV) * sizeof(__nv_bfloat16) +
           (4 * CHUNK + 8 * CHUNK) * sizeof(float);
}

}  // namespace

// Whether keys of dk elements and values of dv take the kernel.
CRANE_API int crane_memory_chunks_supports(int dk, int dv) {
    return dk > 0 && dk % 16 == 0 && dk <= 256 && dv > 0 && dv % 8 == 0 && memory_chunks_smem(dk) <= 220 * 1024;
}

CRANE_API int crane_memory_chunks(const void* proj, int cols, int q_off, int k_off, int v_off, const float* logs, int logs_ld,
                                  const int* cu_q, const int* kv_len, const int* slots, int n_slots, float* state,
                                  long long slot_stride, float* o_raw, float* den, int n_entries, int H, int dk, int dv,
                                  int rows_per_lane, int lanes, float q_scale, int min_len, int* err, cudaStream_t st) {
    if (n_entries <= 0) return 0;
    if (!crane_memory_chunks_supports(dk, dv) || ((cols | q_off | k_off | v_off) & 7) || ((uintptr_t)proj & 15) ||
        ((uintptr_t)o_raw & 7) || rows_per_lane * lanes < dk || min_len < 1)
        return (int)cudaErrorInvalidValue;
    const size_t smem = memory_chunks_smem(dk);
    const auto kern = dk <= 128 ? memory_chunks_kernel<1> : memory_chunks_kernel<2>;
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(memory_chunks_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess ||
            cudaFuncSetAttribute(memory_chunks_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess)
            return (int)cudaGetLastError();
        configured = true;
    }
    return crane_launch(kern, dim3((dv + 1 + CB - 1) / CB, H, n_entries), dim3(256), smem, st, (const __nv_bfloat16*)proj, cols,
                        q_off, k_off, v_off, logs, logs_ld, cu_q, kv_len, slots, n_slots, state, slot_stride, o_raw, den, H, dk,
                        dv, rows_per_lane, lanes, q_scale, min_len, err);
}
