// Linear recurrences with one matrix state S [dk, dv] per head and request, and what surrounds them.
//
//     S <- diag(w_t) S                       (w_t: a decay per key channel, or one number per head)
//     u  = beta_t (v_t - S^T k_t)            (`delta`: the delta rule's correction; else u = v_t)
//     S <- S + k_t u^T
//     o_t = S^T q_t                          (the read-out sees the token's own write)
// or, `bonus`,
//     o_t = S^T r_t + b_t v_t                (the read-out sees the state BEFORE the token's write, and of the
//     S <- diag(w_t) S + k_t v_t^T            token itself only b_t = sum_i r_i u_i k_i, a number per head)
// or, `gated`,
//     S <- w_t S + b_t k_t v_t^T,  N <- w_t N + b_t k_t     (N: one more column of S whose values are 1)
//     o_t = S^T q_t,  den_t = N . q_t                       (divided where the head is normed)
//
// `matrix_state_scan` walks each request's tokens in order.  Columns of S do not talk to one another:
// a CTA holds a block of columns of one (request, head), a column's rows spread over LANES lanes of a
// warp (ROWS rows each, in registers), dot products over the rows finished by shuffles.  The inputs of
// every token (q, k, v, w, beta) are 32-bit rows of an `aux` buffer that a prep kernel writes:
//   * `conv_delta_prep`: q, k, v through a short causal convolution over time and silu, q and k scaled
//     to unit length per head, beta = sigmoid(.), w = exp(-exp(A) softplus(. + dt)) per head (unless a decay
//     per key channel comes from elsewhere); the last taps - 1 inputs of the convolutions are part of the
//     request's state, moved on by the lane that reads them in a step of single tokens, else by
//     `conv_state_update`;
//   * `decay_gate_prep`: q scaled, k, v, and w = sigmoid(z)^(1 / tau) per key channel with z a
//     low-rank product plus bias;
//   * `exp_gate_prep`: q scaled, k, v, and of exponential gates under a running maximum the kept share w, the new
//     token's share b and the floor of the normaliser, per head; the maximum is part of the request's state;
//   * `bonus_prep` (also as further blocks of `low_rank_expand`): r, k, v and the number b per head.
// `token_shift_mix` forms what the projections of the bonus recurrence read, h + (h' - h) mu with h' the
// previous token's row, which is part of the request's state.  `low_rank_expand` is the second matrix of a
// low-rank product with what follows it (a decay, or nothing).
// `head_norm_gate` norms each head's read-out over dv (of a `gated` scan after the division by its normaliser),
// applies the weight and silu(gate) or sigmoid(gate).
// `head_talk_mix` and `pair_norm_mean` belong to attention whose heads exchange their weights and to
// two mixers side by side.
// The state lives in 32-bit in the request's slot, in the order the scan's threads hold it:
// [head][row / LANES][column][row % LANES]; a request whose first token is in the step starts from zero.
#include <type_traits>

#include "common.cuh"

namespace {

__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// ------------------------------------------------------ convolution + delta-rule inputs
// proj row: [q (G d) | k (G d) | v (H dv) | ...] with b (H) at column `b_off` and a (H) at `a_off` (-1: no
// decay is formed here).  aux row: [q (G d) | k (G d) | v (H dv) | ...] with w (H) at `w_off` and beta (H) at
// `beta_off`.  conv_w [2 G d + H dv][taps] float.  conv_state: inside the slot's state
// at `conv_off`, [taps - 1][C].  Grid (tokens, blocks of heads); a warp per head of q, k or v (2 G + H of
// them): a q or k head is written as the convolution left it, then scaled by the same lanes once its
// sum of squares is known.  SINGLE: every entry of the step has one token, so the lane that reads a channel's kept
// inputs is the only one and moves them on.
template <typename T, bool SINGLE>
__global__ void __launch_bounds__(256)
conv_delta_prep_kernel(GemmOut<T> proj, int cols, const int* __restrict__ tok_entry,
                       const int* __restrict__ cu_q, const int* __restrict__ kv_len,
                       const int* __restrict__ slots, int n_slots, const float* __restrict__ state,
                       float* state_out, long long slot_stride, long long conv_off,
                       const float* __restrict__ conv_w, int taps,
                       const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                       float* __restrict__ aux, int aux_cols, int H, int G, int d, int dv, int b_off, int a_off,
                       int w_off, int beta_off, float key_eps, float q_scale, int* err) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int e = tok_entry[t];
    if (e < 0) return;
    const int C = 2 * G * d + H * dv;
    const int first = cu_q[e];
    const int i = t - first;                                         // the token's place in its portion
    const int start = kv_len[e] - (cu_q[e + 1] - first);             // tokens of the request before the step
    const int slot = slots[e];
    if (slot < 0 || slot >= n_slots) {
        if (threadIdx.x == 0 && blockIdx.y == 0) atomicOr(err, CRANE_ERR_SLOT_RANGE);
        return;
    }
    const float* cs = state + (long long)slot * slot_stride + conv_off;
    float* out = aux + (long long)t * aux_cols;
    const int lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    for (int unit = blockIdx.y * nw + (threadIdx.x >> 5); unit < 2 * G + H; unit += gridDim.y * nw) {
        const bool qk = unit < 2 * G;
        const int width = qk ? d : dv;
        const int c_first = qk ? unit * d : 2 * G * d + (unit - 2 * G) * dv;
        float ss = 0.f;
        for (int cc = lane; cc < width; cc += 32) {
            const int c = c_first + cc;
            float acc = 0.f;
            if (SINGLE) {                              // (state_out: the same slots, through a pointer that may be written)
                float* kept = state_out + (long long)slot * slot_stride + conv_off + c;
                for (int j = 0; j < taps; ++j) {
                    float x = 0.f;
                    if (j == taps - 1) x = proj.load((long long)t * cols + c);
                    else if (start - (taps - 1 - j) >= 0) x = kept[(long long)j * C];
                    acc = fmaf(conv_w[(long long)c * taps + j], x, acc);
                    if (j > 0) kept[(long long)(j - 1) * C] = x;
                }
            } else {
                for (int j = 0; j < taps; ++j) {
                    const int back = taps - 1 - j;
                    float x = 0.f;
                    if (i - back >= 0) x = proj.load((long long)(t - back) * cols + c);
                    else if (start + i - back >= 0) x = cs[(long long)(taps - 1 + i - back) * C + c];
                    acc = fmaf(conv_w[(long long)c * taps + j], x, acc);
                }
            }
            const float v = silu_f(acc);
            out[c] = v;
            ss = fmaf(v, v, ss);
        }
        if (qk) {
            ss = warp_sum(ss);
            const float r = rsqrtf(ss + key_eps) * (unit < G ? q_scale : 1.f);
            for (int cc = lane; cc < width; cc += 32) out[c_first + cc] *= r;      // each lane its own elements
        }
    }
    if (blockIdx.y == 0) {
        for (int h = threadIdx.x; h < H; h += blockDim.x) {
            const long long row = (long long)t * cols;
            const float b = proj.load(row + b_off + h);
            if (a_off >= 0) out[w_off + h] = expf(-expf(a_log[h]) * softplus_f(proj.load(row + a_off + h) + dt_bias[h]));
            out[beta_off + h] = 1.f / (1.f + expf(-b));
        }
    }
}

// One thread per (entry, channel): the last taps - 1 inputs of the channel after this step (a step of
// nothing but single tokens has moved them on already).
constexpr int MAX_TAPS = 16;
template <typename T>
__global__ void __launch_bounds__(128)
conv_state_update_kernel(GemmOut<T> proj, int cols, const int* __restrict__ cu_q,
                         const int* __restrict__ kv_len, const int* __restrict__ slots, int n_slots,
                         float* __restrict__ state, long long slot_stride, long long conv_off, int taps, int C) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int first = cu_q[e], q_len = cu_q[e + 1] - first;
    if (q_len <= 0 || c >= C) return;
    const int slot = slots[e];
    if (slot < 0 || slot >= n_slots) return;
    const int end = kv_len[e], start = end - q_len;
    float* cs = state + (long long)slot * slot_stride + conv_off;
    float old[MAX_TAPS];
#pragma unroll
    for (int j = 0; j < MAX_TAPS; ++j) old[j] = (j < taps - 1) ? cs[(long long)j * C + c] : 0.f;
#pragma unroll
    for (int j = 0; j < MAX_TAPS; ++j) {
        if (j < taps - 1) {
            const int p = end - (taps - 1) + j;
            float v = 0.f;
            if (p >= start) v = proj.load((long long)(first + p - start) * cols + c);
            else if (p >= 0) {
                const int k = taps - 1 + p - start;
                float o = 0.f;
#pragma unroll
                for (int m = 0; m < MAX_TAPS; ++m) if (m == k) o = old[m];
                v = o;
            }
            cs[(long long)j * C + c] = v;
        }
    }
}

// ------------------------------------------------------ inputs of the recurrence with a decay per channel
// proj row: [q (H d) | k (H d) | v (H dv) | gate (H dv) | low (rank)].  aux row: [q (H d) | k (H d) |
// v (H dv) | w (H d)].  a2t [rank][H d] float, bias [H d].
template <typename T>
__global__ void __launch_bounds__(256)
decay_gate_prep_kernel(GemmOut<T> proj, int cols, const int* __restrict__ tok_entry,
                       const float* __restrict__ a2t, const float* __restrict__ bias, int rank,
                       float inv_tau, float q_scale, float* __restrict__ aux, int aux_cols, int H, int d, int dv) {
    extern __shared__ float low[];                    // [rank]
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    if (tok_entry[t] < 0) return;
    const int hd = H * d, hv = H * dv;
    const long long row = (long long)t * cols;
    for (int r = threadIdx.x; r < rank; r += blockDim.x) low[r] = proj.load(row + 2 * hd + 2 * hv + r);
    __syncthreads();
    float* out = aux + (long long)t * aux_cols;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < hd; c += gridDim.y * blockDim.x) {
        out[c] = proj.load(row + c) * q_scale;
        out[hd + c] = proj.load(row + hd + c);
        float z = bias[c];
#pragma unroll 8
        for (int r = 0; r < rank; ++r) z = fmaf(low[r], a2t[(long long)r * hd + c], z);
        // sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
        out[2 * hd + hv + c] = expf(-softplus_f(-z) * inv_tau);
    }
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < hv; c += gridDim.y * blockDim.x)
        out[2 * hd + c] = proj.load(row + 2 * hd + c);
}

// ------------------------------------------------------ exponential gates under a running maximum
// proj row: [q (H d) | k (H d) | v (H dv) | ...] with the input gate (H) at column `i_off` and the forget gate (H) at
// `f_off`.  aux row: [q * q_scale | k | v | ...] with w, b and floor (H each) one behind the other at `w_off`:
//     i = cap tanh((z_i + bias_i) / cap),  f = log sigmoid(cap tanh((z_f + bias_f) / cap))
//     M' = max(f + M, i);  w = exp(f + M - M'),  b = exp(i - M'),  floor = exp(-M')
// M (0 before a request's first token) lies in the slot, [H] at `m_off`.  The first `gate_blocks` CTAs work out the
// gates, a CTA per (entry, head), or (SINGLE: every entry of the step has one token) a thread; the others copy q, k and
// v, `by` CTAs a token.  M -> max(M + A, B) composes to maps of the same form, so a CTA takes 1,024 tokens at a time,
// four a thread, and finds the M before every thread's four by a scan over lanes and warps; a thread goes token by
// token, and a token's w is taken from the very M that the token before it left.
// `logs` (or null): for entries of at least `logs_min` tokens, which walk in chunks, log w and log b go to
// [n][2 H] there instead of w and b to aux, and nothing is copied.
template <typename T, bool SINGLE>
__global__ void __launch_bounds__(256)
exp_gate_prep_kernel(GemmOut<T> proj, int cols, const int* __restrict__ tok_entry, const int* __restrict__ cu_q,
                     const int* __restrict__ kv_len, const int* __restrict__ slots, int n_slots,
                     float* __restrict__ state, long long slot_stride, long long m_off,
                     const float* __restrict__ bias_i, const float* __restrict__ bias_f, float cap, float q_scale,
                     float* __restrict__ aux, int aux_cols, int n_entries, int H, int d, int dv, int i_off, int f_off,
                     int w_off, int gate_blocks, int by, float* __restrict__ logs, int logs_min, int* err) {
    pdl_launch_dependents();
    pdl_wait();
    const int hd = H * d, hv = H * dv;
    if ((int)blockIdx.x >= gate_blocks) {
        const int t = ((int)blockIdx.x - gate_blocks) / by, part = ((int)blockIdx.x - gate_blocks) % by;
        const int te = tok_entry[t];
        if (te < 0 || (logs != nullptr && cu_q[te + 1] - cu_q[te] >= logs_min)) return;
        const long long row = (long long)t * cols;
        float* out = aux + (long long)t * aux_cols;
        const int n = 2 * hd + hv;
        if (((cols | aux_cols | hd | n) & 1) == 0) {
            for (int c = 2 * (part * blockDim.x + threadIdx.x); c < n; c += 2 * by * blockDim.x) {
                const float2 v = proj.load2(row + c);
                const float f = c < hd ? q_scale : 1.f;
                st2(out + c, v.x * f, v.y * f);
            }
        } else {
            for (int c = part * blockDim.x + threadIdx.x; c < n; c += by * blockDim.x)
                out[c] = proj.load(row + c) * (c < hd ? q_scale : 1.f);
        }
        return;
    }
    // li = -inf and lf = 0 (past a portion's end) leave M as it is
    auto gates = [&](float zi, float zf, float bi, float bf, float& li, float& lf) {
        const float x = cap * tanhf((zf + bf) / cap);
        li = cap * tanhf((zi + bi) / cap);
        lf = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
    };
    bool as_logs = false;
    auto write = [&](long long t, int h, float li, float lf, float before, float m) {
        float* out = aux + t * aux_cols + w_off + h;
        out[2 * H] = expf(-m);
        if (as_logs) {
            logs[t * 2 * H + h] = lf + before - m;
            logs[t * 2 * H + H + h] = li - m;
            return;
        }
        out[0] = expf(lf + before - m);
        out[H] = expf(li - m);
    };
    const int wid = SINGLE ? (int)(blockIdx.x * blockDim.x + threadIdx.x) : (int)blockIdx.x;
    if (wid >= n_entries * H) return;
    const int e = wid / H, h = wid % H;
    const int first = cu_q[e], q_len = cu_q[e + 1] - first;
    if (q_len <= 0) return;
    const int slot = slots[e];
    if (slot < 0 || slot >= n_slots) {
        if (SINGLE || threadIdx.x == 0) atomicOr(err, CRANE_ERR_SLOT_RANGE);
        return;
    }
    float* kept = state + (long long)slot * slot_stride + m_off + h;
    float m0 = kv_len[e] > q_len ? *kept : 0.f;
    const float bi = bias_i[h], bf = bias_f[h];
    as_logs = logs != nullptr && q_len >= logs_min;
    if (SINGLE) {
        float li, lf;
        const long long row = (long long)first * cols + h;
        gates(proj.load(row + i_off), proj.load(row + f_off), bi, bf, li, lf);
        const float m = fmaxf(lf + m0, li);
        write(first, h, li, lf, m0, m);
        *kept = m;
        return;
    }
    constexpr int PER = 4, WARPS = 8;
    __shared__ float part_a[WARPS], part_b[WARPS], last[WARPS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float zi[PER], zf[PER];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int t = t0 + (int)threadIdx.x * PER + j;
            const long long row = (long long)(first + (t < q_len ? t : q_len - 1)) * cols + h;
            zi[j] = proj.load(row + i_off);
            zf[j] = proj.load(row + f_off);
        }
    };
    fetch(0);
    for (int t0 = 0; t0 < q_len; t0 += WARPS * 32 * PER) {
        const int t = t0 + (int)threadIdx.x * PER;
        float li[PER], lf[PER], m[PER];
        float A = 0.f, B = -INFINITY;
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            gates(zi[j], zf[j], bi, bf, li[j], lf[j]);
            if (t + j >= q_len) li[j] = -INFINITY, lf[j] = 0.f;
            B = fmaxf(B + lf[j], li[j]);
            A += lf[j];
        }
        if (t0 + WARPS * 32 * PER < q_len) fetch(t0 + WARPS * 32 * PER);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pa = __shfl_up_sync(0xffffffffu, A, o), pb = __shfl_up_sync(0xffffffffu, B, o);
            if (lane >= o) {
                B = fmaxf(pb + A, B);
                A += pa;
            }
        }
        if (lane == 31) part_a[warp] = A, part_b[warp] = B;
        const float pa = __shfl_up_sync(0xffffffffu, A, 1), pb = __shfl_up_sync(0xffffffffu, B, 1);
        __syncthreads();
        float run = m0;                                     // M before the warp's tokens, then before the thread's
        for (int w = 0; w < warp; ++w) run = fmaxf(run + part_a[w], part_b[w]);
        if (lane > 0) run = fmaxf(run + pa, pb);
#pragma unroll
        for (int j = 0; j < PER; ++j) m[j] = run = fmaxf(lf[j] + run, li[j]);
        if (lane == 31) last[warp] = m[PER - 1];
        float before = __shfl_up_sync(0xffffffffu, m[PER - 1], 1);
        __syncthreads();
        if (lane == 0) before = warp == 0 ? m0 : last[warp - 1];
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            if (t + j < q_len) write(first + t + j, h, li[j], lf[j], before, m[j]);
            before = m[j];
        }
        m0 = last[WARPS - 1];                               // (`part_a` and `last` are written again behind a barrier that all readers have reached)
    }
    if (threadIdx.x == 0) *kept = m0;
}

// ------------------------------------------------------ what the bonus recurrence's projections read
// out[g][t][c] = h[t][c] + (h'[t][c] - h[t][c]) mu[g][c] for every mix g, h' the row of the request's token before
// (zeros before its first one).  The row before a portion's first token lies in the slot, float [hidden] at
// `row_off`; the thread that reads it there puts the portion's last row in its place.  Grid (tokens, column
// blocks).
template <typename T>
__global__ void __launch_bounds__(256)
token_shift_mix_kernel(const T* __restrict__ h, const float* __restrict__ mu, int mixes,
                       const int* __restrict__ tok_entry, const int* __restrict__ cu_q,
                       const int* __restrict__ kv_len, const int* __restrict__ slots, int n_slots,
                       float* __restrict__ state, long long slot_stride, long long row_off, T* __restrict__ out,
                       long long group_stride, int hidden, int* err) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int e = tok_entry[t];
    if (e < 0) return;
    const int first = cu_q[e], end = cu_q[e + 1];
    const int slot = slots[e];
    if (slot < 0 || slot >= n_slots) {
        if (threadIdx.x == 0 && blockIdx.y == 0) atomicOr(err, CRANE_ERR_SLOT_RANGE);
        return;
    }
    const bool opens = t == first && kv_len[e] == end - first;       // the request's first token
    float* kept = state + (long long)slot * slot_stride + row_off;
    const long long row = (long long)t * hidden;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < hidden; c += gridDim.y * blockDim.x) {
        const float x = to_f32(h[row + c]);
        float before;
        if (t == first) {
            before = opens ? 0.f : kept[c];
            kept[c] = to_f32(h[(long long)(end - 1) * hidden + c]);
        } else {
            before = to_f32(h[row - hidden + c]);
        }
        const float diff = before - x;
        for (int g = 0; g < mixes; ++g)
            out[(long long)g * group_stride + row + c] = from_f32<T>(fmaf(diff, mu[(long long)g * hidden + c], x));
    }
}

// proj row: [r (H d) | k (H d) | v (H dv) | ...].  aux row: [r | k | v | ... ] with b (H) at column `b_off`:
// b = sum_i r_i u_i k_i.  A warp per (token, head).
struct BonusJob { const float* u; float* aux; int aux_cols, b_off, H, d, dv; };     // (u null: no such job)
template <typename T>
__device__ __forceinline__ void bonus_head(const GemmOut<T>& proj, int cols, const BonusJob& job, int t, int h, int lane) {
    const float* u = job.u;
    float* aux = job.aux;
    const int aux_cols = job.aux_cols, b_off = job.b_off, H = job.H, d = job.d, dv = job.dv;
    const long long row = (long long)t * cols;
    float* out = aux + (long long)t * aux_cols;
    const int hd = H * d;
    float b = 0.f;
    if (((cols | d | dv | aux_cols) & 1) == 0) {                              // two neighbours a lane
        for (int c = 2 * lane; c < d; c += 64) {
            const float2 r = proj.load2(row + h * d + c), k = proj.load2(row + hd + h * d + c), uv = ld2(u + h * d + c);
            st2(out + h * d + c, r.x, r.y);
            st2(out + hd + h * d + c, k.x, k.y);
            b = fmaf(r.x * uv.x, k.x, fmaf(r.y * uv.y, k.y, b));
        }
        for (int c = 2 * lane; c < dv; c += 64) {
            const float2 v = proj.load2(row + 2 * hd + h * dv + c);
            st2(out + 2 * hd + h * dv + c, v.x, v.y);
        }
        b = warp_sum(b);
        if (lane == 0) out[b_off + h] = b;
        return;
    }
    for (int c = lane; c < d; c += 32) {
        const float r = proj.load(row + h * d + c), k = proj.load(row + hd + h * d + c);
        out[h * d + c] = r;
        out[hd + h * d + c] = k;
        b = fmaf(r * u[h * d + c], k, b);
    }
    for (int c = lane; c < dv; c += 32) out[2 * hd + h * dv + c] = proj.load(row + 2 * hd + h * dv + c);
    b = warp_sum(b);
    if (lane == 0) out[b_off + h] = b;
}

template <typename T>
__global__ void __launch_bounds__(128)
bonus_prep_kernel(GemmOut<T> proj, int cols, const int* __restrict__ tok_entry, const BonusJob job, int n) {
    pdl_launch_dependents();
    pdl_wait();
    const long long wid = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (wid >= (long long)n * job.H) return;
    const int t = (int)(wid / job.H);
    if (tok_entry[t] >= 0) bonus_head<T>(proj, cols, job, t, (int)(wid % job.H), threadIdx.x & 31);
}

// ------------------------------------------------------ the second matrix of a low-rank product
// z[t][c] = sum_r in(low[t][low_off + r]) w[c][r], in the identity or tanh, then
//   LR_PLAIN       out (T) = z
//   LR_SOFT_DECAY  out (float) = exp(-exp(rate[c / per_rate]) softplus(z + bias[c]))
//   LR_EXP_DECAY   out (float) = exp(-exp(z + bias[c]))
// Up to two such products of one row of `low` (one mixer's decay and gate) are one launch.
enum LowRankKind : int { LR_PLAIN = 0, LR_SOFT_DECAY = 1, LR_EXP_DECAY = 2 };
struct LowRankPart {
    const void* w;                // [n_out][ld_w] (MMA) or [rank][n_out] (FP32 cores), T
    const float* bias;
    const float* rate;
    void* out;
    long long out_ld;
    int low_off, rank, ld_w, n_out, kind, tanh_in, per_rate;
};
// The grid's column blocks: the first part's, the second's up to `col_blocks`, then (if there is one) the bonus job's,
// whose (token, head) pairs of the row tile are dealt out to the warps of those blocks.
struct LowRankArgs { LowRankPart part[2]; int col_blocks0, col_blocks; BonusJob bonus; };
template <typename T>
__device__ __forceinline__ void bonus_blocks(const GemmOut<T>& proj, int cols, const int* __restrict__ tok_entry,
                                             const LowRankArgs& args, int t0, int nt) {
    const int nw = blockDim.x >> 5, H = args.bonus.H;
    const int first = ((int)blockIdx.y - args.col_blocks) * nw + (int)(threadIdx.x >> 5);
    for (int x = first; x < nt * H; x += ((int)gridDim.y - args.col_blocks) * nw) {
        const int t = t0 + x / H;
        if (tok_entry[t] >= 0) bonus_head<T>(proj, cols, args.bonus, t, x % H, threadIdx.x & 31);
    }
}

// What a column adds to z and multiplies the rate by.
struct LowRankColumn { float bias, rate; };
__device__ __forceinline__ LowRankColumn low_rank_column(const LowRankPart& p, int c) {
    LowRankColumn k{0.f, 1.f};
    if (p.kind != LR_PLAIN && c < p.n_out) {
        k.bias = p.bias[c];
        if (p.kind == LR_SOFT_DECAY) k.rate = expf(p.rate[c / p.per_rate]);
    }
    return k;
}
__device__ __forceinline__ float low_rank_decay(const LowRankPart& p, const LowRankColumn& k, float z) {
    z += k.bias;
    return expf(-(p.kind == LR_SOFT_DECAY ? k.rate * softplus_f(z) : expf(z)));
}
template <typename T>
__device__ __forceinline__ void low_rank_store(const LowRankPart& p, const LowRankColumn& k, int t, int c, float z) {
    const long long at = (long long)t * p.out_ld + c;
    if (p.kind == LR_PLAIN) reinterpret_cast<T*>(p.out)[at] = from_f32<T>(z);
    else reinterpret_cast<float*>(p.out)[at] = low_rank_decay(p, k, z);
}

// FP32 cores: a CTA takes 16 tokens and 128 columns, a thread per column; r in order 0 .. rank - 1.
constexpr int LR_TT = 16;
template <typename T>
__global__ void __launch_bounds__(128)
low_rank_simt_kernel(GemmOut<T> low, int cols, const int* __restrict__ tok_entry, const LowRankArgs args, int n) {
    extern __shared__ float xs[];                     // [LR_TT][rank]
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * LR_TT, nt = min(LR_TT, n - t0);
    if ((int)blockIdx.y >= args.col_blocks) return bonus_blocks<T>(low, cols, tok_entry, args, t0, nt);
    const bool second = (int)blockIdx.y >= args.col_blocks0;
    const LowRankPart& p = args.part[second ? 1 : 0];
    for (int i = threadIdx.x; i < LR_TT * p.rank; i += blockDim.x) {
        const int tt = i / p.rank, r = i % p.rank;
        float v = 0.f;
        if (tt < nt && tok_entry[t0 + tt] >= 0) {
            v = low.load((long long)(t0 + tt) * cols + p.low_off + r);
            if (p.tanh_in) v = tanhf(v);
        }
        xs[i] = v;
    }
    __syncthreads();
    const int c = ((int)blockIdx.y - (second ? args.col_blocks0 : 0)) * 128 + threadIdx.x;
    if (c >= p.n_out) return;
    const LowRankColumn col = low_rank_column(p, c);
    const T* w = reinterpret_cast<const T*>(p.w);
    float acc[LR_TT];
#pragma unroll
    for (int tt = 0; tt < LR_TT; ++tt) acc[tt] = 0.f;
    for (int r = 0; r < p.rank; ++r) {
        const float wv = to_f32(w[(long long)r * p.n_out + c]);
#pragma unroll
        for (int tt = 0; tt < LR_TT; ++tt) acc[tt] = fmaf(wv, xs[tt * p.rank + r], acc[tt]);
    }
#pragma unroll
    for (int tt = 0; tt < LR_TT; ++tt)
        if (tt < nt && tok_entry[t0 + tt] >= 0) low_rank_store<T>(p, col, t0 + tt, c, acc[tt]);
}

// Tensor cores (bf16, warp-level MMA), ranks up to 256: a CTA takes 64 tokens (16 per warp) and 64 columns, or
// (FEW: a step of at most 16 tokens) 16 tokens and 64 columns, 16 per warp.  The weights' rows are stored
// `ld_w` = rank rounded up to 16 long, zero-filled.
__device__ __forceinline__ void lr_ldsm_x4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
constexpr int LR_COLS = 64;
template <bool FEW>
__global__ void __launch_bounds__(128)
low_rank_mma_kernel(GemmOut<__nv_bfloat16> low, int cols, const int* __restrict__ tok_entry, const LowRankArgs args,
                    int n) {
    constexpr int BM = FEW ? 16 : 64;
    extern __shared__ __align__(16) unsigned char lr_smem[];
    if ((int)blockIdx.y >= args.col_blocks) {
        pdl_launch_dependents();
        pdl_wait();
        return bonus_blocks<__nv_bfloat16>(low, cols, tok_entry, args, blockIdx.x * BM, min(BM, n - (int)blockIdx.x * BM));
    }
    const bool second = (int)blockIdx.y >= args.col_blocks0;
    const LowRankPart& p = args.part[second ? 1 : 0];
    const int ld = p.ld_w + 8;
    __nv_bfloat16* a_s = reinterpret_cast<__nv_bfloat16*>(lr_smem);      // [BM][ld]
    __nv_bfloat16* w_s = a_s + BM * ld;                                   // [64][ld]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    const int t0 = blockIdx.x * BM;
    const int c0 = ((int)blockIdx.y - (second ? args.col_blocks0 : 0)) * LR_COLS;
    pdl_launch_dependents();
    // the weights depend on no earlier kernel
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w);
    const int pieces = p.ld_w >> 3;
    for (int i = threadIdx.x; i < LR_COLS * pieces; i += blockDim.x) {
        const int r = i / pieces, q = i % pieces;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (c0 + r < p.n_out) v = *reinterpret_cast<const uint4*>(w + (long long)(c0 + r) * p.ld_w + q * 8);
        *reinterpret_cast<uint4*>(w_s + r * ld + q * 8) = v;
    }
    pdl_wait();
#pragma unroll 4
    for (int tt = warp; tt < BM; tt += 4) {
        const bool ok = t0 + tt < n && tok_entry[t0 + tt] >= 0;
        const long long at = (long long)(t0 + tt) * cols + p.low_off;
        for (int r = lane; r < p.ld_w; r += 32) {
            float v = 0.f;
            if (ok && r < p.rank) {
                v = low.load(at + r);
                if (p.tanh_in) v = tanhf(v);
            }
            a_s[tt * ld + r] = __float2bfloat16_rn(v);
        }
    }
    __syncthreads();
    const int wrow = FEW ? 0 : warp * 16;
    constexpr int NB = FEW ? 2 : 8;                   // blocks of 8 columns a warp takes
    const int wcol = FEW ? warp * 16 : 0;
    float acc[NB][4];
#pragma unroll
    for (int i = 0; i < NB; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int ks = 0; ks < (p.ld_w >> 4); ++ks) {
        uint32_t a0, a1, a2, a3;
        lr_ldsm_x4(a0, a1, a2, a3, a_s + (wrow + (lane & 15)) * ld + ks * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int j = 0; j < NB / 2; ++j) {
            uint32_t b0, b1, b2, b3;
            lr_ldsm_x4(b0, b1, b2, b3, w_s + (wcol + j * 16 + (lane & 7) + (lane >> 4) * 8) * ld + ks * 16 + ((lane >> 3) & 1) * 8);
            asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                         : "+f"(acc[2 * j][0]), "+f"(acc[2 * j][1]), "+f"(acc[2 * j][2]), "+f"(acc[2 * j][3])
                         : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
            asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                         : "+f"(acc[2 * j + 1][0]), "+f"(acc[2 * j + 1][1]), "+f"(acc[2 * j + 1][2]), "+f"(acc[2 * j + 1][3])
                         : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b2), "r"(b3));
        }
    }
    const int ta = t0 + wrow + g;
    bool live[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) live[half] = ta + 8 * half < n && tok_entry[ta + 8 * half] >= 0;
    // two neighbouring columns a store where rows are evenly long and the first element is aligned
    const bool pairs = (p.out_ld & 1) == 0 && ((uintptr_t)p.out & 7) == 0;
#pragma unroll
    for (int i = 0; i < NB; ++i) {
        const int c = c0 + wcol + i * 8 + 2 * t4;
        if (c >= p.n_out) continue;
        const LowRankColumn ka = low_rank_column(p, c), kb = low_rank_column(p, c + 1);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            if (!live[half]) continue;
            const int t = ta + 8 * half;
            const float za = acc[i][2 * half], zb = acc[i][2 * half + 1];
            if (pairs && c + 1 < p.n_out) {
                const long long at = (long long)t * p.out_ld + c;
                if (p.kind == LR_PLAIN) st2(reinterpret_cast<__nv_bfloat16*>(p.out) + at, za, zb);
                else st2(reinterpret_cast<float*>(p.out) + at, low_rank_decay(p, ka, za), low_rank_decay(p, kb, zb));
            } else {
                low_rank_store<__nv_bfloat16>(p, ka, t, c, za);
                if (c + 1 < p.n_out) low_rank_store<__nv_bfloat16>(p, kb, t, c + 1, zb);
            }
        }
    }
}

// ------------------------------------------------------ the recurrence
// grid (entries, heads, column blocks); block = COLS columns x LANES lanes.  aux offsets: q_off, k_off,
// v_off, w_off, beta_off (the delta rule's beta, or the bonus b); q/k head of head h is h / qk_rep; w is [H d]
// (w_vec) or [H].  o_raw float [n][H dv].
// Tokens come in tiles of `tile_tokens` whose vectors all threads copy into shared memory with 4-byte
// asynchronous copies, the next tile while the current one is walked: a tile's fetch from DRAM is as
// long as walking several tokens, and the walk must not wait for it.
__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src)
                 : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src)
                 : "memory");
}
constexpr int SCAN_TOKENS = 16;
// The sum over the LANES (a power of two, aligned in the warp) that share a column; LANES 0: `lanes` at run
// time.
template <int LANES>
__device__ __forceinline__ float lanes_sum(float x, int lanes) {
    if (LANES > 0) {
#pragma unroll
        for (int o = LANES >> 1; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
        return x;
    }
    if (lanes > 16) x += __shfl_xor_sync(0xffffffffu, x, 16);
    if (lanes > 8) x += __shfl_xor_sync(0xffffffffu, x, 8);
    if (lanes > 4) x += __shfl_xor_sync(0xffffffffu, x, 4);
    if (lanes > 2) x += __shfl_xor_sync(0xffffffffu, x, 2);
    if (lanes > 1) x += __shfl_xor_sync(0xffffffffu, x, 1);
    return x;
}
// A lane holds ROWS neighbouring rows of its column.  FULL: the lanes' rows are exactly the dk rows; no row
// is tested and a lane reads its part of a vector 16 bytes at a time.  WVEC: a decay per row (else one per
// head).  MODE: what a token does (plain, the delta rule's correction, bonus, gated: there column dv is the normaliser, whose read-out goes
// to `den`).  LANES: the lanes of a column when the kernel is compiled for
// them (0: any).  The first `walkers` threads walk the tokens; one more warp does nothing but copy the next
// tile of tokens into shared memory meanwhile, since a walking warp's time is its instructions per token.
enum ScanMode : int { SCAN_PLAIN = 0, SCAN_DELTA = 1, SCAN_BONUS = 2, SCAN_GATED = 3 };
template <int ROWS, bool FULL, int MODE, bool WVEC, int LANES>
__global__ void __launch_bounds__(288)
matrix_state_scan_kernel(const float* __restrict__ aux, int aux_cols, int q_off, int k_off, int v_off, int w_off,
                         int beta_off, int qk_rep, const int* __restrict__ cu_q,
                         const int* __restrict__ kv_len, const int* __restrict__ slots, int n_slots,
                         float* __restrict__ state, long long slot_stride, float* __restrict__ o_raw,
                         int H, int dk, int dv, int lanes_rt, int cols_per_block, int tile_tokens, int vec4,
                         int walkers, float* __restrict__ den, int max_len, int* err) {
    constexpr bool DELTA = MODE == SCAN_DELTA, BONUS = MODE == SCAN_BONUS, GATED = MODE == SCAN_GATED;
    const int dvt = dv + (GATED ? 1 : 0);             // columns of the state
    extern __shared__ __align__(16) float tile[];     // two tiles of [tile_tokens][3 dk + cols + 2, to a multiple of 4]
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x, h = blockIdx.y;
    const int first = cu_q[e], q_len = cu_q[e + 1] - first;
    if (q_len <= 0 || (max_len > 0 && q_len >= max_len)) return;      // (long entries may be another kernel's)
    const int slot = slots[e];
    if (slot < 0 || slot >= n_slots) {
        if (threadIdx.x == 0) atomicOr(err, CRANE_ERR_SLOT_RANGE);
        return;
    }
    const int lanes = LANES > 0 ? LANES : lanes_rt;
    const int start = kv_len[e] - q_len;
    const int hq = h / qk_rep;
    const int stride = (3 * dk + cols_per_block + 2 + 3) & ~3;       // rows start on 16 bytes
    const int c0 = blockIdx.z * cols_per_block;
    const int tile_floats = tile_tokens * stride;
    const int n_tiles = (q_len + tile_tokens - 1) / tile_tokens;
    const bool producer = (int)threadIdx.x >= walkers;

    // ---- the copying warp: a token's vectors are runs of its row; units of 16 bytes (`vec4`: every run starts
    // on 16 bytes and is a multiple of them) or of 4
    const int wl = threadIdx.x & 31;
    const int unit = vec4 ? 4 : 1;
    const int nq = dk / unit, nvu = max(0, min(cols_per_block, dv - c0)) / unit;
    const int n_units = (WVEC ? 3 : 2) * nq + nvu;
    auto place = [&](int x, int& so, int& dofs) {                    // unit x of a token: where from, where to
        if (x < nq) so = q_off + hq * dk + x * unit, dofs = x * unit;
        else if (x < 2 * nq) so = k_off + hq * dk + (x - nq) * unit, dofs = dk + (x - nq) * unit;
        else if (WVEC && x < 3 * nq) so = w_off + h * dk + (x - 2 * nq) * unit, dofs = 2 * dk + (x - 2 * nq) * unit;
        else {
            const int y = x - (WVEC ? 3 : 2) * nq;
            so = v_off + h * dv + c0 + y * unit, dofs = 3 * dk + y * unit;
        }
    };
    auto copy = [&](float* dst, const float* src) {
        if (vec4) cp_async16(dst, src);
        else cp_async4(dst, src);
    };
    int so0 = -1, do0 = 0, so1 = -1, do1 = 0;                         // the lane's first two units, the same for every token
    if (producer) {
        if (wl < n_units) place(wl, so0, do0);
        if (wl + 32 < n_units) place(wl + 32, so1, do1);
    }
    auto fetch = [&](int t0, float* buf) {
        const int nt = min(tile_tokens, q_len - t0);
        const float* a = aux + (long long)(first + t0) * aux_cols;
        float* b = buf;
        for (int tt = 0; tt < nt; ++tt, a += aux_cols, b += stride) {
            if (so0 >= 0) copy(b + do0, a + so0);
            if (so1 >= 0) copy(b + do1, a + so1);
            for (int x = wl + 64; x < n_units; x += 32) {
                int so, dofs;
                place(x, so, dofs);
                copy(b + dofs, a + so);
            }
            if (wl == 0) {
                if (WVEC) b[3 * dk + cols_per_block] = 1.f;
                else cp_async4(b + 3 * dk + cols_per_block, a + w_off + h);
            } else if (wl == 1) {
                if (DELTA || BONUS || GATED) cp_async4(b + 3 * dk + cols_per_block + 1, a + beta_off + h);
                else b[3 * dk + cols_per_block + 1] = 1.f;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 0;" ::: "memory");
    };
    if (producer) fetch(0, tile);

    // ---- the walkers
    const int lane = threadIdx.x % lanes, cl = threadIdx.x / lanes;
    const int r0 = lane * ROWS;                       // the lane's rows: r0 .. r0 + ROWS - 1
    const int col = c0 + cl;
    const bool live = !producer && cl < cols_per_block && col < dvt;
    const bool idle = !__any_sync(0xffffffffu, live);   // (a warp without a column walks nothing)
    const int vcol = live ? cl : 0;
    // state [H][ROWS][columns][lanes]
    float* sp = state + (long long)slot * slot_stride + (long long)h * ROWS * dvt * lanes;
    float s[ROWS];
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
        s[i] = (live && start > 0 && (FULL || r0 + i < dk)) ? sp[((long long)i * dvt + col) * lanes + lane] : 0.f;
    __syncthreads();                                  // the first tile is there
    const bool norm_col = GATED && col == dv;
    const long long o_step = norm_col ? H : (long long)H * dv;
    for (int it = 0; it < n_tiles; ++it) {
        const int t0 = it * tile_tokens;
        const int nt = min(tile_tokens, q_len - t0);
        if (producer) {
            if (it + 1 < n_tiles) fetch(t0 + tile_tokens, tile + ((it + 1) & 1) * tile_floats);
        } else if (!idle) {
            const float* tp = tile + (it & 1) * tile_floats;
            float* op = (norm_col ? den + h : o_raw + h * dv + (live ? col : 0)) + (long long)(first + t0) * o_step;
#pragma unroll(ROWS == 8 ? 2 : 1)
            for (int tt = 0; tt < nt; ++tt, tp += stride, op += o_step) {
                float qv[ROWS], kv[ROWS], wv[ROWS];
                if (FULL) {                            // lane's rows are one aligned run of each vector
#pragma unroll
                    for (int i = 0; i < ROWS; i += 4) {
                        const float4 a4 = *reinterpret_cast<const float4*>(tp + r0 + i);
                        const float4 b4 = *reinterpret_cast<const float4*>(tp + dk + r0 + i);
                        qv[i] = a4.x, qv[i + 1] = a4.y, qv[i + 2] = a4.z, qv[i + 3] = a4.w;
                        kv[i] = b4.x, kv[i + 1] = b4.y, kv[i + 2] = b4.z, kv[i + 3] = b4.w;
                        if (WVEC) {
                            const float4 c4 = *reinterpret_cast<const float4*>(tp + 2 * dk + r0 + i);
                            wv[i] = c4.x, wv[i + 1] = c4.y, wv[i + 2] = c4.z, wv[i + 3] = c4.w;
                        }
                    }
                } else {                               // rows past dk: zeros, and their state stays zero
#pragma unroll
                    for (int i = 0; i < ROWS; ++i) {
                        const bool in = r0 + i < dk;
                        qv[i] = in ? tp[r0 + i] : 0.f;
                        kv[i] = in ? tp[dk + r0 + i] : 0.f;
                        if (WVEC) wv[i] = in ? tp[2 * dk + r0 + i] : 0.f;
                    }
                }
                const float vv = tp[3 * dk + vcol];    // a column that is not live reads a neighbour's and writes nothing
                const float ws = WVEC ? 1.f : tp[3 * dk + cols_per_block];
                if (BONUS) {
                    float rd = 0.f;
#pragma unroll
                    for (int i = 0; i < ROWS; ++i) {
                        rd = fmaf(s[i], qv[i], rd);
                        s[i] = fmaf(s[i], WVEC ? wv[i] : ws, kv[i] * vv);
                    }
                    rd = lanes_sum<LANES>(rd, lanes);
                    if (live && lane == 0) *op = fmaf(tp[3 * dk + cols_per_block + 1], vv, rd);
                    continue;
                }
                float dot = 0.f;
#pragma unroll
                for (int i = 0; i < ROWS; ++i) {
                    s[i] *= WVEC ? wv[i] : ws;
                    if (DELTA) dot = fmaf(s[i], kv[i], dot);
                }
                float u = vv;
                if (GATED) u = tp[3 * dk + cols_per_block + 1] * (norm_col ? 1.f : vv);
                if (DELTA) {
                    dot = lanes_sum<LANES>(dot, lanes);
                    u = tp[3 * dk + cols_per_block + 1] * (vv - dot);
                }
                float rd = 0.f;
#pragma unroll
                for (int i = 0; i < ROWS; ++i) {
                    s[i] = fmaf(kv[i], u, s[i]);
                    rd = fmaf(s[i], qv[i], rd);
                }
                rd = lanes_sum<LANES>(rd, lanes);
                if (live && lane == 0) *op = rd;
            }
        }
        __syncthreads();              // the next tile is there for all; all have left this one
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i) sp[((long long)i * dvt + col) * lanes + lane] = s[i];
    }
}

// ------------------------------------------------------ head norm and gate
// out[t][h dv + c] = o_raw / rms_over_dv(o_raw) * norm_w[h norm_step + c] * act(gate[t][gate_off + h dv + c]),
// norm_step 0 (a weight that the heads share) or dv, act silu or, `sigmoid_gate`, sigmoid; a warp per
// (token, head).  `den` [n][H] (or null): o_raw is first divided by max(|den|, floor) + den_eps, floor of token t at
// floor_at[t * floor_ld + h].
template <typename T>
__global__ void __launch_bounds__(128)
head_norm_gate_kernel(const float* __restrict__ o_raw, GemmOut<T> proj, int cols, int gate_off,
                      const int* __restrict__ tok_entry, const float* __restrict__ norm_w, int norm_step,
                      int sigmoid_gate, float eps, const float* __restrict__ den, const float* __restrict__ floor_at,
                      int floor_ld, float den_eps, T* __restrict__ out, int n, int H, int dv) {
    pdl_launch_dependents();
    pdl_wait();
    const long long wid = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (wid >= (long long)n * H) return;
    const int t = (int)(wid / H), h = (int)(wid % H);
    if (tok_entry[t] < 0) return;
    const float* o = o_raw + ((long long)t * H + h) * dv;
    // the read-out's own normaliser, if it has one, divides it first
    const float inv = den == nullptr ? 1.f
                                     : 1.f / (fmaxf(fabsf(den[(long long)t * H + h]), floor_at[(long long)t * floor_ld + h]) + den_eps);
    if (((dv | cols | gate_off) & 1) == 0 && (norm_step & 1) == 0) {          // heads of even size: two neighbours a lane
        const long long gp = (long long)t * cols + gate_off + h * dv;
        float2 v[4], gv[4];                                                   // (the first 256 elements stay in registers)
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 2 * lane + 64 * i;
            if (c < dv) {
                v[i] = ld2(o + c);
                gv[i] = proj.load2(gp + c);
                ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, ss));
            }
        }
        for (int c = 2 * lane + 256; c < dv; c += 64) {
            const float2 a = ld2(o + c);
            ss = fmaf(a.x, a.x, fmaf(a.y, a.y, ss));
        }
        ss = warp_sum(ss);
        const float rstd = inv * rsqrtf(ss * inv * inv / (float)dv + eps);
        auto act = [&](float g) { return sigmoid_gate ? 1.f / (1.f + expf(-g)) : silu_f(g); };
        const float* w = norm_w + h * norm_step;
        T* dst = out + ((long long)t * H + h) * dv;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 2 * lane + 64 * i;
            if (c < dv) st2(dst + c, v[i].x * rstd * w[c] * act(gv[i].x), v[i].y * rstd * w[c + 1] * act(gv[i].y));
        }
        for (int c = 2 * lane + 256; c < dv; c += 64) {
            const float2 a = ld2(o + c), g = proj.load2(gp + c);
            st2(dst + c, a.x * rstd * w[c] * act(g.x), a.y * rstd * w[c + 1] * act(g.y));
        }
        return;
    }
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) { const float v = o[c]; ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    const float rstd = inv * rsqrtf(ss * inv * inv / (float)dv + eps);
    for (int c = lane; c < dv; c += 32) {
        const float g = proj.load((long long)t * cols + gate_off + h * dv + c);
        const float a = sigmoid_gate ? 1.f / (1.f + expf(-g)) : silu_f(g);
        out[((long long)t * H + h) * dv + c] = from_f32<T>(o[c] * rstd * norm_w[h * norm_step + c] * a);
    }
}

// ------------------------------------------------------ heads that exchange their weights
// cross [n][H][G][dv] float: query head g's softmax weights applied to the values of every key/value
// head.  out[t][h] = sum_g talk[h][g] cross[t][g][h / (H / G)].  Grid (tokens, heads).
template <typename T>
__global__ void __launch_bounds__(128)
head_talk_mix_kernel(const float* __restrict__ cross, const float* __restrict__ talk,
                     const int* __restrict__ tok_entry, T* __restrict__ out, int H, int G, int dv, int out_head) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, h = blockIdx.y;
    if (tok_entry[t] < 0) return;
    const int rep = H / G;
    for (int c = threadIdx.x; c < out_head; c += blockDim.x) {               // out_head <= dv columns are kept
        const float* src = cross + ((long long)t * H * G + h / rep) * dv + c;
        float acc = 0.f;
        for (int g = 0; g < H; ++g) acc = fmaf(talk[h * H + g], src[(long long)g * G * dv], acc);
        out[((long long)t * H + h) * out_head + c] = from_f32<T>(acc);
    }
}

// ------------------------------------------------------ two mixers side by side
// out = (a / rms(a) * wa + b / rms(b) * wb) / 2 over the width; a CTA per row.
// Four neighbours of a product (aligned), all slices' loads in flight eight at a time, added in slice order.
template <typename T>
__device__ __forceinline__ float4 load4(const GemmOut<T>& g, long long idx) {
    if (g.parts == nullptr) {
        const float2 a = ld2(g.whole + idx), b = ld2(g.whole + idx + 2);
        return make_float4(a.x, a.y, b.x, b.y);
    }
    float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i = 0; i < g.n_parts; i += 8) {
        float4 q[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
            q[j] = i + j < g.n_parts ? *(const float4*)(g.parts + (long long)(i + j) * g.part_stride + idx)
                                     : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < 8; ++j) d.x += q[j].x, d.y += q[j].y, d.z += q[j].z, d.w += q[j].w;
    }
    return make_float4(to_f32(from_f32<T>(d.x)), to_f32(from_f32<T>(d.y)), to_f32(from_f32<T>(d.z)), to_f32(from_f32<T>(d.w)));
}
template <typename T>
__global__ void __launch_bounds__(1024)
pair_norm_mean_kernel(GemmOut<T> a, GemmOut<T> b, const float* __restrict__ wa, const float* __restrict__ wb,
                      float eps, T* __restrict__ out, int hidden, int quad) {
    extern __shared__ float row2[];                   // [2 hidden]
    __shared__ float scratch[32];
    pdl_launch_dependents();
    const long long base = (long long)blockIdx.x * hidden;
    float sa = 0.f, sb = 0.f;
    // Rows of four columns a thread: everything a thread reads is in flight at once, the weights before the wait for
    // the kernel before, and stays in its registers.
    if (quad) {
        const int c = threadIdx.x * 4;
        const bool in = c < hidden;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 va = in ? *(const float4*)(wa + c) : zero, vb = in ? *(const float4*)(wb + c) : zero;
        pdl_wait();
        const float4 x = in ? load4(a, base + c) : zero, y = in ? load4(b, base + c) : zero;
        sa = block_sum((x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w), scratch);
        sb = block_sum((y.x * y.x + y.y * y.y) + (y.z * y.z + y.w * y.w), scratch);
        const float ra = rsqrtf(sa / (float)hidden + eps), rb = rsqrtf(sb / (float)hidden + eps);
        if (in) {
            st2(out + base + c, 0.5f * (x.x * ra * va.x + y.x * rb * vb.x), 0.5f * (x.y * ra * va.y + y.y * rb * vb.y));
            st2(out + base + c + 2, 0.5f * (x.z * ra * va.z + y.z * rb * vb.z), 0.5f * (x.w * ra * va.w + y.w * rb * vb.w));
        }
        return;
    }
    pdl_wait();
    const bool pairs = (hidden & 1) == 0;             // rows of even length: two neighbours a load and a store
    if (pairs) {
        for (int c = 2 * threadIdx.x; c < hidden; c += 2 * blockDim.x) {
            const float2 x = a.load2(base + c), y = b.load2(base + c);
            row2[c] = x.x, row2[c + 1] = x.y;
            row2[hidden + c] = y.x, row2[hidden + c + 1] = y.y;
            sa = fmaf(x.x, x.x, fmaf(x.y, x.y, sa));
            sb = fmaf(y.x, y.x, fmaf(y.y, y.y, sb));
        }
    } else {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
            const float x = a.load(base + c), y = b.load(base + c);
            row2[c] = x;
            row2[hidden + c] = y;
            sa = fmaf(x, x, sa);
            sb = fmaf(y, y, sb);
        }
    }
    sa = block_sum(sa, scratch);
    sb = block_sum(sb, scratch);
    const float ra = rsqrtf(sa / (float)hidden + eps), rb = rsqrtf(sb / (float)hidden + eps);
    if (pairs) {
        for (int c = 2 * threadIdx.x; c < hidden; c += 2 * blockDim.x)
            st2(out + base + c, 0.5f * (row2[c] * ra * wa[c] + row2[hidden + c] * rb * wb[c]),
                0.5f * (row2[c + 1] * ra * wa[c + 1] + row2[hidden + c + 1] * rb * wb[c + 1]));
    } else {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x)
            out[base + c] = from_f32<T>(0.5f * (row2[c] * ra * wa[c] + row2[hidden + c] * rb * wb[c]));
    }
}

}  // namespace

CRANE_API int crane_conv_delta_prep(int dtype, const void* proj, const float* proj_parts, int n_parts,
                                    long long part_stride, int cols, const int* tok_entry, const int* cu_q,
                                    const int* kv_len, const int* slots, int n_slots, float* state,
                                    long long slot_stride, long long conv_off, const float* conv_w, int taps,
                                    const float* a_log, const float* dt_bias, float* aux, int aux_cols,
                                    int n_tokens, int n_entries, int H, int G, int d, int dv, int b_off, int a_off,
                                    int w_off, int beta_off, float key_eps, float q_scale, int all_single, int* err,
                                    cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    const int C = 2 * G * d + H * dv;
    if (taps < 1 || taps > MAX_TAPS) return (int)cudaErrorInvalidValue;
    // a warp per head; with few tokens the heads spread over more CTAs
    const int units = 2 * G + H;
    int by = (units + 7) / 8;
    while (by > 1 && (long long)n_tokens * by > 4 * 148) by = (by + 1) / 2;
    DISPATCH_T(dtype, {
        GemmOut<T> p{(const T*)proj, proj_parts, n_parts, part_stride};
        const auto kern = all_single ? conv_delta_prep_kernel<T, true> : conv_delta_prep_kernel<T, false>;
        int rc = crane_launch(kern, dim3(n_tokens, by), dim3(256), 0, st, p, cols, tok_entry,
                              cu_q, kv_len, slots, n_slots, (const float*)state, state, slot_stride, conv_off, conv_w,
                              taps, a_log, dt_bias, aux, aux_cols, H, G, d, dv, b_off, a_off, w_off, beta_off, key_eps,
                              q_scale, err);
        if (rc != 0 || taps == 1 || all_single) return rc;
        return crane_launch(conv_state_update_kernel<T>, dim3((C + 127) / 128, n_entries), dim3(128), 0, st, p,
                            cols, cu_q, kv_len, slots, n_slots, state, slot_stride, conv_off, taps, C);
    });
}

CRANE_API int crane_decay_gate_prep(int dtype, const void* proj, const float* proj_parts, int n_parts,
                                    long long part_stride, int cols, const int* tok_entry, const float* a2t,
                                    const float* bias, int rank, float inv_tau, float q_scale, float* aux,
                                    int aux_cols, int n_tokens, int H, int d, int dv, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (rank < 0 || rank > 8192) return (int)cudaErrorInvalidValue;
    DISPATCH_T(dtype, {
        GemmOut<T> p{(const T*)proj, proj_parts, n_parts, part_stride};
        int by = (H * (d > dv ? d : dv) + 255) / 256;            // with few tokens the channels spread over more CTAs
        while (by > 1 && (long long)n_tokens * by > 4 * 148) by = (by + 1) / 2;
        return crane_launch(decay_gate_prep_kernel<T>, dim3(n_tokens, by), dim3(256), (size_t)(rank > 0 ? rank : 1) * 4,
                            st, p, cols, tok_entry, a2t, bias, rank, inv_tau, q_scale, aux, aux_cols, H, d, dv);
    });
}

CRANE_API int crane_exp_gate_prep(int dtype, const void* proj, const float* proj_parts, int n_parts,
                                  long long part_stride, int cols, const int* tok_entry, const int* cu_q,
                                  const int* kv_len, const int* slots, int n_slots, float* state,
                                  long long slot_stride, long long m_off, const float* bias_i, const float* bias_f,
                                  float cap, float q_scale, float* aux, int aux_cols, int n_tokens, int n_entries,
                                  int H, int d, int dv, int i_off, int f_off, int w_off, int all_single, float* logs,
                                  int logs_min, int* err, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    const int gate_blocks = all_single ? (n_entries * H + 255) / 256 : n_entries * H;
    int by = (2 * H * d + H * dv + 511) / 512;               // with few tokens a token's columns spread over more CTAs
    while (by > 1 && (long long)n_tokens * by > 4 * 148) by = (by + 1) / 2;
    DISPATCH_T(dtype, {
        GemmOut<T> p{(const T*)proj, proj_parts, n_parts, part_stride};
        const auto kern = all_single ? exp_gate_prep_kernel<T, true> : exp_gate_prep_kernel<T, false>;
        // (one entry that walks in chunks, whatever padding of less than 64 rows the step has: nothing to copy)
        const int copies = logs != nullptr && n_entries == 1 && n_tokens >= logs_min + 64 ? 0 : n_tokens * by;
        return crane_launch(kern, dim3(gate_blocks + copies), dim3(256), 0, st, p, cols,
                            tok_entry, cu_q, kv_len, slots, n_slots, state, slot_stride, m_off, bias_i, bias_f, cap,
                            q_scale, aux, aux_cols, n_entries, H, d, dv, i_off, f_off, w_off, gate_blocks, by, logs, logs_min, err);
    });
}

CRANE_API int crane_token_shift_mix(int dtype, const void* h, const float* mu, int mixes, const int* tok_entry,
                                    const int* cu_q, const int* kv_len, const int* slots, int n_slots,
                                    float* state, long long slot_stride, long long row_off, void* out,
                                    long long group_stride, int n_tokens, int hidden, int* err, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    int by = (hidden + 255) / 256;
    while (by > 1 && (long long)n_tokens * by > 4 * 148) by = (by + 1) / 2;
    DISPATCH_T(dtype, return crane_launch(token_shift_mix_kernel<T>, dim3(n_tokens, by), dim3(256), 0, st, (const T*)h,
                                          mu, mixes, tok_entry, cu_q, kv_len, slots, n_slots, state, slot_stride,
                                          row_off, (T*)out, group_stride, hidden, err));
}

CRANE_API int crane_bonus_prep(int dtype, const void* proj, const float* proj_parts, int n_parts,
                               long long part_stride, int cols, const int* tok_entry, const float* u, float* aux,
                               int aux_cols, int b_off, int n_tokens, int H, int d, int dv, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    const long long warps = (long long)n_tokens * H;
    DISPATCH_T(dtype, {
        GemmOut<T> p{(const T*)proj, proj_parts, n_parts, part_stride};
        const BonusJob job{u, aux, aux_cols, b_off, H, d, dv};
        return crane_launch(bonus_prep_kernel<T>, dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, st, p, cols,
                            tok_entry, job, n_tokens);
    });
}

// `mma` 1: bf16, weights [n_out][ld_w] with ld_w a multiple of 16 and at most 256, zero-filled behind the rank,
// 16-byte aligned; 0: weights [rank][n_out] on the FP32 cores.  A second part with n_out2 = 0 is absent.
CRANE_API int crane_low_rank_expand(int dtype, const void* low, const float* low_parts, int n_parts,
                                    long long part_stride, int cols, const int* tok_entry, int mma,
                                    const void* w1, const float* bias1, const float* rate1, int per_rate1,
                                    void* out1, long long out_ld1, int low_off1, int rank1, int ld_w1, int n_out1,
                                    int kind1, int tanh1, const void* w2, const float* bias2, const float* rate2,
                                    int per_rate2, void* out2, long long out_ld2, int low_off2, int rank2, int ld_w2,
                                    int n_out2, int kind2, int tanh2, const float* bonus_u, float* bonus_aux,
                                    int bonus_aux_cols, int bonus_off, int bonus_H, int bonus_d, int bonus_dv,
                                    int n_tokens, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    LowRankArgs a;
    a.bonus = BonusJob{bonus_u, bonus_aux, bonus_aux_cols, bonus_off, bonus_H, bonus_d, bonus_dv};
    auto bonus_count = [&](int rows_per_tile) {              // blocks for the bonus job: about a pair a warp, 64 at most
        if (bonus_u == nullptr) return 0;
        const int blocks = ((n_tokens < rows_per_tile ? n_tokens : rows_per_tile) * bonus_H + 3) / 4;
        return blocks < 64 ? blocks : 64;
    };
    a.part[0] = LowRankPart{w1, bias1, rate1, out1, out_ld1, low_off1, rank1, ld_w1, n_out1, kind1, tanh1, per_rate1 > 0 ? per_rate1 : 1};
    a.part[1] = LowRankPart{w2, bias2, rate2, out2, out_ld2, low_off2, rank2, ld_w2, n_out2, kind2, tanh2, per_rate2 > 0 ? per_rate2 : 1};
    int widest = rank1;
    if (n_out2 > 0 && rank2 > widest) widest = rank2;
    if (mma) {
        int ldm = ld_w1;
        for (int i = 0; i < (n_out2 > 0 ? 2 : 1); ++i) {
            const LowRankPart& p = a.part[i];
            if (dtype != 1 || p.ld_w < p.rank || p.ld_w % 16 || p.ld_w <= 0 || p.ld_w > 256 || ((uintptr_t)p.w & 15))
                return (int)cudaErrorInvalidValue;
            if (p.ld_w > ldm) ldm = p.ld_w;
        }
        const int b0 = (n_out1 + LR_COLS - 1) / LR_COLS, b1 = n_out2 > 0 ? (n_out2 + LR_COLS - 1) / LR_COLS : 0;
        a.col_blocks0 = b0;
        a.col_blocks = b0 + b1;
        const bool few = n_tokens <= 16;
        const int bm = few ? 16 : 64;
        const size_t smem = (size_t)(bm + LR_COLS) * (ldm + 8) * sizeof(__nv_bfloat16);
        auto kern = few ? low_rank_mma_kernel<true> : low_rank_mma_kernel<false>;
        static bool attr_set = false;
        if (!attr_set) {
            cudaFuncSetAttribute(low_rank_mma_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 80 * 1024);
            cudaFuncSetAttribute(low_rank_mma_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 80 * 1024);
            attr_set = true;
        }
        GemmOut<__nv_bfloat16> l{(const __nv_bfloat16*)low, low_parts, n_parts, part_stride};
        return crane_launch(kern, dim3((n_tokens + bm - 1) / bm, b0 + b1 + bonus_count(bm)), dim3(128), smem, st, l, cols,
                            tok_entry, a, n_tokens);
    }
    const int b0 = (n_out1 + 127) / 128, b1 = n_out2 > 0 ? (n_out2 + 127) / 128 : 0;
    a.col_blocks0 = b0;
    a.col_blocks = b0 + b1;
    const size_t smem = (size_t)LR_TT * (widest > 0 ? widest : 1) * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    DISPATCH_T(dtype, {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(low_rank_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        GemmOut<T> l{(const T*)low, low_parts, n_parts, part_stride};
        return crane_launch(low_rank_simt_kernel<T>, dim3((n_tokens + LR_TT - 1) / LR_TT, b0 + b1 + bonus_count(LR_TT)), dim3(128),
                            smem, st, l, cols, tok_entry, a, n_tokens);
    });
}

// The scan's geometry for a key size: (rows per lane, lanes per column); 0 rows: too wide.
CRANE_API int crane_matrix_state_plan(int dk, int* rows, int* lanes) {
    int r = dk <= 256 ? 8 : 16, l = 1;
    while (l * r < dk && l < 32) l *= 2;
    if (l * r < dk) { *rows = 0; *lanes = 0; return 1; }
    *rows = r;
    *lanes = l;
    return 0;
}

CRANE_API int crane_matrix_state_scan(const float* aux, int aux_cols, int q_off, int k_off, int v_off, int w_off,
                                      int beta_off, int w_vec, int mode, int qk_rep, const int* cu_q,
                                      const int* kv_len, const int* slots, int n_slots, float* state,
                                      long long slot_stride, float* o_raw, float* den, int n_entries, int H, int dk,
                                      int dv, int max_len, int* err, cudaStream_t st) {
    if (n_entries <= 0) return 0;
    int rows, lanes;
    if (crane_matrix_state_plan(dk, &rows, &lanes) || dv <= 0 || qk_rep <= 0 || mode < 0 || mode > 3 ||
        (mode == SCAN_BONUS && !w_vec) || (mode == SCAN_GATED && (w_vec || den == nullptr)))
        return (int)cudaErrorInvalidValue;
    int cpb = 256 / lanes;
    if (cpb > dv) cpb = dv;
    // few entries and heads: narrower blocks of columns, so that more SMs walk (a column's result does not
    // depend on the block it is in)
    while ((long long)n_entries * H * ((dv + cpb - 1) / cpb) < 148 && cpb > 8) cpb /= 2;
    const int blocks = (dv + (mode == SCAN_GATED ? 1 : 0) + cpb - 1) / cpb;
    const int walkers = ((cpb * lanes + 31) / 32) * 32;        // and a warp that copies
    const size_t per_token = (size_t)((3 * dk + cpb + 2 + 3) & ~3) * sizeof(float);
    const int vec4 = (dk % 4 == 0 && dv % 4 == 0 && cpb % 4 == 0 && aux_cols % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 &&
                      v_off % 4 == 0 && (!w_vec || w_off % 4 == 0) && (uintptr_t)aux % 16 == 0) ? 1 : 0;
    int tile_tokens = (int)((48 * 1024) / (2 * per_token));
    if (tile_tokens > SCAN_TOKENS) tile_tokens = SCAN_TOKENS;
    if (tile_tokens < 1) return (int)cudaErrorInvalidValue;
    const size_t smem = 2 * (size_t)tile_tokens * per_token;
    const bool full = rows * lanes == dk;
    using Kern = decltype(&matrix_state_scan_kernel<8, true, SCAN_DELTA, true, 0>);
    const bool delta = mode == SCAN_DELTA;
    auto pick = [&](auto rows_c, auto lanes_c) -> Kern {
        constexpr int R = decltype(rows_c)::value, L = decltype(lanes_c)::value;
        if (mode == SCAN_BONUS)
            return full ? matrix_state_scan_kernel<R, true, SCAN_BONUS, true, L> : matrix_state_scan_kernel<R, false, SCAN_BONUS, true, 0>;
        if (mode == SCAN_GATED)
            return full ? matrix_state_scan_kernel<R, true, SCAN_GATED, false, L> : matrix_state_scan_kernel<R, false, SCAN_GATED, false, 0>;
        if (full) return delta ? (w_vec ? matrix_state_scan_kernel<R, true, SCAN_DELTA, true, L> : matrix_state_scan_kernel<R, true, SCAN_DELTA, false, L>)
                               : (w_vec ? matrix_state_scan_kernel<R, true, SCAN_PLAIN, true, L> : matrix_state_scan_kernel<R, true, SCAN_PLAIN, false, L>);
        return delta ? (w_vec ? matrix_state_scan_kernel<R, false, SCAN_DELTA, true, 0> : matrix_state_scan_kernel<R, false, SCAN_DELTA, false, 0>)
                     : (w_vec ? matrix_state_scan_kernel<R, false, SCAN_PLAIN, true, 0> : matrix_state_scan_kernel<R, false, SCAN_PLAIN, false, 0>);
    };
    using std::integral_constant;
    Kern kern;
    if (rows != 8) kern = pick(integral_constant<int, 16>{}, integral_constant<int, 0>{});
    else if (full && lanes == 4) kern = pick(integral_constant<int, 8>{}, integral_constant<int, 4>{});      // heads of 32,
    else if (full && lanes == 8) kern = pick(integral_constant<int, 8>{}, integral_constant<int, 8>{});      // 64
    else if (full && lanes == 16) kern = pick(integral_constant<int, 8>{}, integral_constant<int, 16>{});    // and 128
    else kern = pick(integral_constant<int, 8>{}, integral_constant<int, 0>{});
    return crane_launch(kern, dim3(n_entries, H, blocks), dim3(walkers + 32), smem, st, aux, aux_cols, q_off, k_off,
                        v_off, w_off, beta_off, qk_rep, cu_q, kv_len, slots, n_slots, state, slot_stride,
                        o_raw, H, dk, dv, lanes, cpb, tile_tokens, vec4, walkers, den, max_len, err);
}

CRANE_API int crane_head_norm_gate(int dtype, const float* o_raw, const void* proj, const float* proj_parts,
                                   int n_parts, long long part_stride, int cols, int gate_off,
                                   const int* tok_entry, const float* norm_w, int norm_step, int sigmoid_gate,
                                   float eps, const float* den, const float* floor_at, int floor_ld, float den_eps,
                                   void* out, int n_tokens, int H, int dv, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    const long long warps = (long long)n_tokens * H;
    DISPATCH_T(dtype, {
        GemmOut<T> p{(const T*)proj, proj_parts, n_parts, part_stride};
        return crane_launch(head_norm_gate_kernel<T>, dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, st, o_raw, p,
                            cols, gate_off, tok_entry, norm_w, norm_step, sigmoid_gate, eps, den, floor_at, floor_ld, den_eps,
                            (T*)out, n_tokens, H, dv);
    });
}

CRANE_API int crane_head_talk_mix(int dtype, const float* cross, const float* talk, const int* tok_entry, void* out,
                                  int n_tokens, int H, int G, int dv, int out_head, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (G <= 0 || H % G || out_head > dv) return (int)cudaErrorInvalidValue;
    DISPATCH_T(dtype, return crane_launch(head_talk_mix_kernel<T>, dim3(n_tokens, H), dim3(out_head > 64 ? 128 : 64), 0, st, cross, talk,
                                          tok_entry, (T*)out, H, G, dv, out_head));
}

CRANE_API int crane_pair_norm_mean(int dtype, const void* a, const float* a_parts, int an, long long astr,
                                   const void* b, const float* b_parts, int bn, long long bstr, const float* wa,
                                   const float* wb, float eps, void* out, int n_rows, int hidden, cudaStream_t st) {
    if (n_rows <= 0) return 0;
    const size_t smem = (size_t)2 * hidden * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    DISPATCH_T(dtype, {
        GemmOut<T> ga{(const T*)a, a_parts, an, astr};
        GemmOut<T> gb{(const T*)b, b_parts, bn, bstr};
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(pair_norm_mean_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        const int quad = hidden % 4 == 0 && hidden <= 4096 && ((astr | bstr) & 3) == 0 &&
                         (((uintptr_t)wa | (uintptr_t)wb | (uintptr_t)a_parts | (uintptr_t)b_parts) & 15) == 0 &&
                         (((uintptr_t)a | (uintptr_t)b | (uintptr_t)out) & 7) == 0;
        const int threads = quad ? (hidden / 4 + 31) / 32 * 32 : 256;
        return crane_launch(pair_norm_mean_kernel<T>, dim3(n_rows), dim3(threads), quad ? 0 : smem, st, ga, gb, wa, wb, eps,
                            (T*)out, hidden, quad);
    });
}
