// Two recurrent mixers whose state is a matrix per head, and what feeds them.
//
// Delta rule with a decay per key channel (per head, key channels d < D, value channels j < Dv, token by token):
//     S[d][j] <- g_t[d] * S[d][j]
//     u[j]     = beta_t * (v_t[j] - sum_d S[d][j] * k_t[d])
//     S[d][j] <- S[d][j] + k_t[d] * u[j]
//     o_t[j]   = sum_d S[d][j] * q_t[d]                      (the read-out sees the token's own write)
// The same with ONE decay per head, worked out here from its projection a_t, g_t = exp(-exp(A_log) * softplus(a_t + dt_bias)).
// Time mix with a bonus for the current token (value channels j < D as well):
//     o_t[j]   = sum_d r_t[d] * (S[d][j] + u[d] * k_t[d] * v_t[j])
//     S[d][j] <- w_t[d] * S[d][j] + k_t[d] * v_t[j]
// Both run in float32 on a state that lives in the request's slot of a state tensor between steps, [D][Dv] per
// head, so the result at a token depends on the request's tokens up to it and on nothing else: not on how they
// were cut into steps, not on the batch around them.
//
// The delta rule's q, k and v pass a short causal convolution over time per channel and silu, and q and k are
// made unit vectors per head (short_conv_kernel); the last taps - 1 inputs of the convolution are state too.  The
// time mix reads, per projection, x_t + (x_{t-1} - x_t) * mu (token_shift_kernel); x of the last token is state.
#include "common.cuh"

// ------------------------------------------------------------------------------------------ short convolution
// in [T][C] (row stride in_stride) holds the inputs of C channels: first n_unit_heads heads of `unit_dim`
// channels whose outputs are made unit vectors (x / sqrt(sum x^2 + unit_eps)), the first q_heads of them also
// times q_scale; the rest is left as silu gives it.  y[t][c] = silu(sum_j w[c][j] * in[t - (taps-1) + j][c]);
// rows before the request's first row of this step come from tail[slot][taps-1][C] (the inputs that ended the
// step before; zero at the start of a request).  One block per token.
__global__ __launch_bounds__(256) void short_conv_kernel(
    const float* __restrict__ in, long long in_stride, const float* __restrict__ w, int taps,
    const float* __restrict__ state, long long slot_stride, long long tail_off, int max_slots,
    const int32_t* __restrict__ req_of_token, const int32_t* __restrict__ cu_tokens, const int32_t* __restrict__ state_slots,
    int num_reqs, float* __restrict__ out, int C, int n_unit_heads, int q_heads, int unit_dim, float unit_eps,
    float q_scale, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float s_y[];                 // [C]
    const int t = blockIdx.x;
    const int req = req_of_token[t];
    if (req < 0) return;
    if (req >= num_reqs) { if (threadIdx.x == 0) atomicOr(err, AIRUN_DEV_BAD_REQ); return; }
    const int slot = state_slots[req];
    if (slot < 0 || slot >= max_slots) { if (threadIdx.x == 0) atomicOr(err, AIRUN_DEV_BAD_REQ); return; }
    const int i = t - cu_tokens[req];              // place of the token within its request's rows of this step
    const float* tail = state + (size_t)slot * slot_stride + tail_off;
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
        float acc = 0.0f;
        for (int j = 0; j < taps; ++j) {
            const int src = i - (taps - 1) + j;
            const float xv = src >= 0 ? in[(size_t)(t - (taps - 1) + j) * in_stride + c] : tail[(size_t)(i + j) * C + c];
            acc = fmaf(w[(size_t)c * taps + j], xv, acc);
        }
        s_y[c] = acc / (1.0f + expf(-acc));
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
    for (int h = warp; h < n_unit_heads; h += nwarp) {
        float ss = 0.0f;
        for (int d = lane; d < unit_dim; d += 32) { const float v = s_y[h * unit_dim + d]; ss = fmaf(v, v, ss); }
        ss = warp_sum(ss);
        const float inv = (1.0f / sqrtf(ss + unit_eps)) * (h < q_heads ? q_scale : 1.0f);
        for (int d = lane; d < unit_dim; d += 32) out[(size_t)t * C + h * unit_dim + d] = s_y[h * unit_dim + d] * inv;
    }
    for (int c = n_unit_heads * unit_dim + threadIdx.x; c < C; c += blockDim.x) out[(size_t)t * C + c] = s_y[c];
}

// The same for 1 to 4 taps and everything in multiples of four on 16-byte boundaries.  A warp takes one unit (a head that is
// made a unit vector, or 128 * NV of the remaining channels) of TOK consecutive rows of the batch, a lane four neighbouring
// channels (NV times): the rows the tokens read are loaded at once, each of them once for all the taps it serves, and the
// weights, which no kernel writes, before the kernel in front has finished.
template <int TAPS, int NV, int TOK>
__global__ __launch_bounds__(128) void short_conv_rows_kernel(
    const float* __restrict__ in, long long in_stride, const float* __restrict__ w, const float* __restrict__ state,
    long long slot_stride, long long tail_off, int max_slots, const int32_t* __restrict__ req_of_token,
    const int32_t* __restrict__ cu_tokens, const int32_t* __restrict__ state_slots, int num_reqs, float* __restrict__ out, int T,
    int C, int n_unit_heads, int q_heads, int unit_dim, float unit_eps, float q_scale, int* __restrict__ err) {
    pdl_trigger();
    const int lane = threadIdx.x & 31, unit = blockIdx.y * 4 + (threadIdx.x >> 5), t0 = blockIdx.x * TOK;
    const bool is_head = unit < n_unit_heads;
    const int c0 = is_head ? unit * unit_dim : n_unit_heads * unit_dim + (unit - n_unit_heads) * 128 * NV;
    const int width = is_head ? unit_dim : min(128 * NV, C - c0);
    if (width <= 0) return;
    float wt[NV][4][TAPS];
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < TAPS; ++j) wt[v][e][j] = 4 * lane + 128 * v < width ? w[(size_t)(c0 + 4 * lane + 128 * v + e) * TAPS + j] : 0.0f;
    pdl_wait();
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    // rows t0 - (TAPS-1) .. t0 + TOK - 1; those ahead of the first token's request are not read
    const int first_req = req_of_token[t0];
    const int i0 = first_req >= 0 && first_req < num_reqs ? t0 - cu_tokens[first_req] : 0;
    float4 x[TAPS - 1 + TOK][NV];
#pragma unroll
    for (int m = 0; m < TAPS - 1 + TOK; ++m) {
        const int row = t0 - (TAPS - 1) + m;
        const bool on = row < T && (m >= TAPS - 1 || i0 >= TAPS - 1 - m);
#pragma unroll
        for (int v = 0; v < NV; ++v)
            x[m][v] = on && 4 * lane + 128 * v < width ? *reinterpret_cast<const float4*>(in + (size_t)row * in_stride + c0 + 4 * lane + 128 * v) : zero;
    }
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
        const int t = t0 + k;
        if (t >= T) return;
        const int req = req_of_token[t];
        if (req < 0) continue;
        const int slot = req < num_reqs ? state_slots[req] : -1;
        if (slot < 0 || slot >= max_slots) {
            if (lane == 0) atomicOr(err, AIRUN_DEV_BAD_REQ);
            continue;
        }
        const int i = t - cu_tokens[req];
        const float* tail = state + (size_t)slot * slot_stride + tail_off;
        float4 y[NV];
        float ss = 0.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const bool on = 4 * lane + 128 * v < width;
            float4 acc = zero;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                float4 xv = x[k + j][v];
                if (i < TAPS - 1 - j) xv = on ? *reinterpret_cast<const float4*>(tail + (size_t)(i + j) * C + c0 + 4 * lane + 128 * v) : zero;
                acc.x = fmaf(wt[v][0][j], xv.x, acc.x); acc.y = fmaf(wt[v][1][j], xv.y, acc.y);
                acc.z = fmaf(wt[v][2][j], xv.z, acc.z); acc.w = fmaf(wt[v][3][j], xv.w, acc.w);
            }
            acc.x = acc.x / (1.0f + expf(-acc.x)); acc.y = acc.y / (1.0f + expf(-acc.y));
            acc.z = acc.z / (1.0f + expf(-acc.z)); acc.w = acc.w / (1.0f + expf(-acc.w));
            y[v] = acc;
            ss = fmaf(acc.x, acc.x, fmaf(acc.y, acc.y, fmaf(acc.z, acc.z, fmaf(acc.w, acc.w, ss))));
        }
        const float inv = is_head ? (1.0f / sqrtf(warp_sum(ss) + unit_eps)) * (unit < q_heads ? q_scale : 1.0f) : 1.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v)
            if (4 * lane + 128 * v < width)
                *reinterpret_cast<float4*>(out + (size_t)t * C + c0 + 4 * lane + 128 * v) = make_float4(y[v].x * inv, y[v].y * inv, y[v].z * inv, y[v].w * inv);
    }
}

AIRUN_EXPORT int airun_short_conv(const float* in, long long in_stride, const float* w, int taps, const float* state,
                                  long long slot_stride, long long tail_off, int max_slots, const int32_t* req_of_token,
                                  const int32_t* cu_tokens, const int32_t* state_slots, int num_reqs, float* out, int T, int C,
                                  int n_unit_heads, int q_heads, int unit_dim, float unit_eps, float q_scale, int* err,
                                  cudaStream_t stream) {
    if (T < 0 || C <= 0 || taps <= 0 || taps > 64 || in_stride < C || !state || !err || n_unit_heads < 0 || unit_dim <= 0 ||
        (long long)n_unit_heads * unit_dim > C || C > 48 * 1024 / 4)
        return AIRUN_ERR_ARG;
    if (T == 0) return AIRUN_OK;
    const bool vec = taps <= 4 && C % 4 == 0 && in_stride % 4 == 0 && slot_stride % 4 == 0 && tail_off % 4 == 0 && unit_dim % 4 == 0 &&
                     unit_dim <= 256 && (((uintptr_t)in | (uintptr_t)state | (uintptr_t)out) & 15) == 0;
    if (vec) {
        const int nv = n_unit_heads > 0 && unit_dim > 128 ? 2 : 1;
        const dim3 units(1, ceil_div_i(n_unit_heads + ceil_div_i(C - n_unit_heads * unit_dim, 128 * nv), 4));
#define SC_LAUNCH(TAPS, NV, TOK) \
        airun_launch(short_conv_rows_kernel<TAPS, NV, TOK>, dim3(ceil_div_i(T, TOK), units.y), dim3(128), 0, stream, in, in_stride, w, state, \
                     slot_stride, tail_off, max_slots, req_of_token, cu_tokens, state_slots, num_reqs, out, T, C, n_unit_heads, q_heads, \
                     unit_dim, unit_eps, q_scale, err)
#define SC_TOK(TAPS) do { if (nv == 2) SC_LAUNCH(TAPS, 2, 2); else if (T <= 128) SC_LAUNCH(TAPS, 1, 1); else SC_LAUNCH(TAPS, 1, 8); } while (0)
        if (taps == 1) SC_TOK(1);
        else if (taps == 2) SC_TOK(2);
        else if (taps == 3) SC_TOK(3);
        else SC_TOK(4);
#undef SC_TOK
#undef SC_LAUNCH
        return airun_launch_status();
    }
    airun_launch(short_conv_kernel, dim3(T), dim3(256), (size_t)C * sizeof(float), stream, in, in_stride, w, taps, state, slot_stride,
                 tail_off, max_slots, req_of_token, cu_tokens, state_slots, num_reqs, out, C, n_unit_heads, q_heads, unit_dim,
                 unit_eps, q_scale, err);
    return airun_launch_status();
}

// ------------------------------------------------------------------------------------------ token shift
// out[s][t][c] = x[t][c] + (prev[c] - x[t][c]) * mu[s][c] for s < n_mix, in the type of `out`; prev is x[t-1], or,
// for the first row a request brings in this step, the row its state keeps (zero at the start of a request).
template <typename TOut>
__global__ __launch_bounds__(256) void token_shift_kernel(
    const float* __restrict__ x, const float* __restrict__ mu, int n_mix, const float* __restrict__ state,
    long long slot_stride, long long prev_off, int max_slots, const int32_t* __restrict__ req_of_token,
    const int32_t* __restrict__ cu_tokens, const int32_t* __restrict__ state_slots, int num_reqs, TOut* __restrict__ out,
    int T, int W, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const int req = req_of_token[t];
    if (req < 0) return;
    if (req >= num_reqs) { if (threadIdx.x == 0) atomicOr(err, AIRUN_DEV_BAD_REQ); return; }
    const int slot = state_slots[req];
    if (slot < 0 || slot >= max_slots) { if (threadIdx.x == 0) atomicOr(err, AIRUN_DEV_BAD_REQ); return; }
    const float* prev = t > cu_tokens[req] ? x + (size_t)(t - 1) * W : state + (size_t)slot * slot_stride + prev_off;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        const float xv = x[(size_t)t * W + c], d = prev[c] - xv;
        for (int s = 0; s < n_mix; ++s)
            out[((size_t)s * T + t) * W + c] = from_f32<TOut>(fmaf(d, mu[(size_t)s * W + c], xv));
    }
}

AIRUN_EXPORT int airun_token_shift(const float* x, const float* mu, int n_mix, const float* state, long long slot_stride,
                                   long long prev_off, int max_slots, const int32_t* req_of_token, const int32_t* cu_tokens,
                                   const int32_t* state_slots, int num_reqs, void* out, int out_dtype, int T, int W, int* err,
                                   cudaStream_t stream) {
    if (T < 0 || W <= 0 || n_mix <= 0 || !state || !err) return AIRUN_ERR_ARG;
    if (T == 0) return AIRUN_OK;
    if (out_dtype == AIRUN_DT_F32)
        airun_launch(token_shift_kernel<float>, dim3(T), dim3(256), 0, stream, x, mu, n_mix, state, slot_stride, prev_off, max_slots,
                     req_of_token, cu_tokens, state_slots, num_reqs, (float*)out, T, W, err);
    else if (out_dtype == AIRUN_DT_BF16)
        airun_launch(token_shift_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, x, mu, n_mix, state, slot_stride, prev_off,
                     max_slots, req_of_token, cu_tokens, state_slots, num_reqs, (__nv_bfloat16*)out, T, W, err);
    else
        return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// ------------------------------------------------------------------------------------------ the recurrences
// One block per (request, head, 128 / DG value columns), 128 threads.  A value column is shared by DG = 4 or 8
// neighbouring lanes, each of which keeps NS key channels of the column's state in registers for the whole step: the
// sums over key channels are NS multiply-adds in a thread and two or three shuffles, and nothing but the state chains
// one token to the next.  The key channels of a lane are every DG-th group of four, so the lanes of a column read
// neighbouring float4 of the token's q, k and decay from shared memory.  (Eight lanes a column from 33 key channels
// on: what bounds a prompt is the chain of its tokens, and a warp's instructions per token halve.)  Tokens are staged through shared memory
// a few at a time by asynchronous copies into one of two stages.  The blocks of a request also move its small state on, a
// share of the channels each: the last inputs of the short convolution (delta rule) or the last token's x (time mix).
#define RS_TT 16
#define RS_DELTA 0
#define RS_WKV 1
#define RS_DELTA_HEAD 2

struct RecurrentArgs {
    const float* q; const float* k; const float* v; const float* g;     // delta: q, k, v, decay; time mix: r, k, v, decay
    long long q_stride, k_stride, v_stride, g_stride;                    // row strides in elements
    const float* beta; long long beta_stride;                            // delta: [T][heads], before its sigmoid
    const float* a_log; const float* dt_bias;                            // delta with one decay per head: [heads] each, and g is a_t [T][heads]
    const float* bonus;                                                  // time mix: [heads][D]
    float* state; long long slot_stride; int max_slots;
    const int32_t* cu_tokens; const int32_t* state_slots;
    float* out;                                                          // [T][heads * Dv]
    int heads, kv_rep, D, Dv;                                            // head h reads q/k head h / kv_rep
    // the small state, moved on by all blocks of the request
    const float* tail_src; long long tail_src_stride; long long tail_off; int tail_rows, tail_width;
    int* err;
};

// The request's small state: its last `tail_rows` rows become the last rows of (what it held, then this step's rows).  A
// thread owns whole columns; row s comes from a later row, so a batch of rows that is read before it is written, in
// ascending order, never reads what was written.
__device__ __forceinline__ void rs_move_tail(const RecurrentArgs& a, int slot, int t0, int n) {
    if (a.tail_rows <= 0) return;
    float* tail = a.state + (size_t)slot * a.slot_stride + a.tail_off;
    const int R = a.tail_rows, Wd = a.tail_width, share = blockIdx.y * gridDim.z + blockIdx.z;
    for (int c = share * blockDim.x + threadIdx.x; c < Wd; c += blockDim.x * gridDim.y * gridDim.z) {
        for (int s0 = 0; s0 < R; s0 += 4) {
            float v[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int src = s0 + i + n;
                v[i] = s0 + i >= R ? 0.0f : src < R ? tail[(size_t)src * Wd + c] : a.tail_src[(size_t)(t0 + src - R) * a.tail_src_stride + c];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (s0 + i < R) tail[(size_t)(s0 + i) * Wd + c] = v[i];
        }
    }
}

__device__ __forceinline__ void rs_cp4(float* smem, const float* gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void rs_cp16(float* smem, const float* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}

template <int MODE, int NS, int DG>
__global__ __launch_bounds__(128) void recurrent_state_kernel(RecurrentArgs a) {
    pdl_trigger();
    pdl_wait();
    constexpr int DP = NS * DG;
    constexpr int COLS = 128 / DG;               // value columns of a block: 32 / DG a warp
    constexpr int TT = DP >= 256 ? 4 : DP >= 128 ? 8 : RS_TT;     // tokens of a stage (static shared memory stays under 48 KB)
    // two stages: the next tokens arrive by asynchronous copies while these are used
    constexpr bool DELTA = MODE != RS_WKV, HEAD = MODE == RS_DELTA_HEAD;
    constexpr int GW = HEAD ? 1 : DP;            // decays of a token: one number, or one a key channel
    __shared__ __align__(16) float s_q[2][TT][DP], s_k[2][TT][DP], s_g[2][TT][GW], s_v[2][TT][COLS];
    __shared__ float s_b[2][TT], s_kq[HEAD ? TT : 1];
    const int r = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * COLS;
    const int t0 = a.cu_tokens[r], n = a.cu_tokens[r + 1] - t0;
    if (n <= 0) return;
    const int slot = a.state_slots[r];
    if (slot < 0 || slot >= a.max_slots) {
        if (threadIdx.x == 0) atomicOr(a.err, AIRUN_DEV_BAD_REQ);
        return;
    }
    const int D = a.D, Dv = a.Dv;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int dg = lane & (DG - 1), cl = warp * (32 / DG) + lane / DG, col = col0 + cl;
    const bool col_ok = col < Dv;
    const int qk_head = head / a.kv_rep;
    const int ncol = min(COLS, Dv - col0);
    // the padding beyond D and Dv is zero in both stages and is never copied into (nothing to do when there is none)
    if (D < DP || ncol < COLS) {
        for (int e = threadIdx.x; e < 2 * TT * DP; e += 128) { (&s_q[0][0][0])[e] = 0.0f; (&s_k[0][0][0])[e] = 0.0f; }
        for (int e = threadIdx.x; e < 2 * TT * GW; e += 128) (&s_g[0][0][0])[e] = 0.0f;
        for (int e = threadIdx.x; e < 2 * TT * COLS; e += 128) (&s_v[0][0][0])[e] = 0.0f;
        __syncthreads();
    }
    const float* qh = a.q + (size_t)qk_head * D;
    const float* kh = a.k + (size_t)qk_head * D;
    const float* gh = a.g + (size_t)head * (HEAD ? 1 : D);
    const float* vh = a.v + (size_t)head * Dv + col0;
    const bool vec = (D % 4 == 0) && ((a.q_stride | a.k_stride | (HEAD ? 0 : a.g_stride)) % 4 == 0) &&
                     ((((uintptr_t)qh | (uintptr_t)kh | (HEAD ? 0 : (uintptr_t)gh)) & 15) == 0);
    const bool vvec = (ncol % 4 == 0) && (a.v_stride % 4 == 0) && (((uintptr_t)vh & 15) == 0);
    auto stage = [&](int base, int buf) {
        const int nt = min(TT, n - base);
        if (vec) {
            const int per = D / 4;
            for (int e = threadIdx.x; e < nt * per; e += 128) {
                const int tt = e / per, d = (e - tt * per) * 4;
                const size_t row = (size_t)(t0 + base + tt);
                rs_cp16(&s_q[buf][tt][d], qh + row * a.q_stride + d);
                rs_cp16(&s_k[buf][tt][d], kh + row * a.k_stride + d);
                if (!HEAD) rs_cp16(&s_g[buf][tt][HEAD ? 0 : d], gh + row * a.g_stride + d);
            }
        } else {
            for (int e = threadIdx.x; e < nt * D; e += 128) {
                const int tt = e / D, d = e - tt * D;
                const size_t row = (size_t)(t0 + base + tt);
                rs_cp4(&s_q[buf][tt][d], qh + row * a.q_stride + d);
                rs_cp4(&s_k[buf][tt][d], kh + row * a.k_stride + d);
                if (!HEAD) rs_cp4(&s_g[buf][tt][HEAD ? 0 : d], gh + row * a.g_stride + d);
            }
        }
        if (vvec) {
            const int per = ncol / 4;
            for (int e = threadIdx.x; e < nt * per; e += 128) {
                const int tt = e / per, c = (e - tt * per) * 4;
                rs_cp16(&s_v[buf][tt][c], vh + (size_t)(t0 + base + tt) * a.v_stride + c);
            }
        } else {
            for (int e = threadIdx.x; e < nt * ncol; e += 128) {
                const int tt = e / ncol, c = e - tt * ncol;
                rs_cp4(&s_v[buf][tt][c], vh + (size_t)(t0 + base + tt) * a.v_stride + c);
            }
        }
        if (DELTA && threadIdx.x < nt)
            rs_cp4(&s_b[buf][threadIdx.x], a.beta + (size_t)(t0 + base + threadIdx.x) * a.beta_stride + head);
        if (HEAD && threadIdx.x < nt) rs_cp4(&s_g[buf][threadIdx.x][0], gh + (size_t)(t0 + base + threadIdx.x) * a.g_stride);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    float* sbase = a.state + (size_t)slot * a.slot_stride + (size_t)head * D * Dv + (col_ok ? col : 0);
    // channel of register i: group of four (i / 4) * DG + dg, element i % 4
    float S[NS], bonus[MODE == RS_WKV ? NS : 1];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int d = ((i >> 2) * DG + dg) * 4 + (i & 3);
        S[i] = (col_ok && d < D) ? sbase[(size_t)d * Dv] : 0.0f;
        if (MODE == RS_WKV) bonus[i] = d < D ? a.bonus[(size_t)head * D + d] : 0.0f;
    }
    float* orow = a.out + (size_t)t0 * ((size_t)a.heads * Dv) + (size_t)head * Dv + col;
    const float rate = HEAD ? expf(a.a_log[head]) : 0.0f, dt = HEAD ? a.dt_bias[head] : 0.0f;
    int it = 0;
    for (int base = 0; base < n; base += TT, ++it) {
        const int buf = it & 1, nt = min(TT, n - base);
        if (base + TT < n) {
            stage(base + TT, buf ^ 1);          // that stage was last read before the barrier that ended the iteration before
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        if (HEAD) {
            // what belongs to a token and not to a column, once for the stage: its beta, its decay and k . q
            constexpr int TPT = 128 / TT;       // neighbouring threads that share a token
            const int tt = threadIdx.x / TPT, e0 = threadIdx.x % TPT;
            float kq = 0.0f;
#pragma unroll
            for (int d = e0; d < DP; d += TPT) kq = fmaf(s_k[buf][tt][d], s_q[buf][tt][d], kq);
#pragma unroll
            for (int off = 1; off < TPT; off <<= 1) kq += __shfl_xor_sync(0xffffffffu, kq, off);
            if (e0 == 0 && tt < nt) {
                const float z = s_g[buf][tt][0] + dt;
                s_g[buf][tt][0] = expf(-rate * (fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)))));
                s_b[buf][tt] = 1.0f / (1.0f + expf(-s_b[buf][tt]));
                s_kq[tt] = kq;
            }
            __syncthreads();
        }
#pragma unroll 2
        for (int tt = 0; tt < nt; ++tt) {
            const float vj = s_v[buf][tt][cl];
            float o;
            if (HEAD) {
                // the decay is one number, so it is applied to the sums over the old state and in the update
                const float gt = s_g[buf][tt][0], beta = s_b[buf][tt];
                float pred[2] = {0.0f, 0.0f}, oq[2] = {0.0f, 0.0f}, kr[NS];
#pragma unroll
                for (int i4 = 0; i4 < NS / 4; ++i4) {
                    const int d = (i4 * DG + dg) * 4;
                    const float4 k4 = *reinterpret_cast<const float4*>(&s_k[buf][tt][d]);
                    const float4 q4 = *reinterpret_cast<const float4*>(&s_q[buf][tt][d]);
                    const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        kr[4 * i4 + e] = kk[e];
                        pred[e & 1] = fmaf(S[4 * i4 + e], kk[e], pred[e & 1]);
                        oq[e & 1] = fmaf(S[4 * i4 + e], qq[e], oq[e & 1]);
                    }
                }
                float p = pred[0] + pred[1], oqs = oq[0] + oq[1];
#pragma unroll
                for (int off = 1; off < DG; off <<= 1) {
                    p += __shfl_xor_sync(0xffffffffu, p, off);
                    oqs += __shfl_xor_sync(0xffffffffu, oqs, off);
                }
                const float u = beta * fmaf(-gt, p, vj);
#pragma unroll
                for (int i = 0; i < NS; ++i) S[i] = fmaf(kr[i], u, gt * S[i]);
                o = fmaf(u, s_kq[tt], gt * oqs);
            } else if (MODE == RS_DELTA) {
                // beta arrives as the projection's output: the gate is its sigmoid
                const float beta = 1.0f / (1.0f + expf(-s_b[buf][tt]));
                float pred[2] = {0.0f, 0.0f}, oq[2] = {0.0f, 0.0f}, kq[2] = {0.0f, 0.0f};
#pragma unroll
                for (int i4 = 0; i4 < NS / 4; ++i4) {
                    const int d = (i4 * DG + dg) * 4;
                    const float4 g4 = *reinterpret_cast<const float4*>(&s_g[buf][tt][HEAD ? 0 : d]);
                    const float4 k4 = *reinterpret_cast<const float4*>(&s_k[buf][tt][d]);
                    const float4 q4 = *reinterpret_cast<const float4*>(&s_q[buf][tt][d]);
                    const float gg[4] = {g4.x, g4.y, g4.z, g4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float sd = gg[e] * S[4 * i4 + e];
                        S[4 * i4 + e] = sd;
                        pred[e & 1] = fmaf(sd, kk[e], pred[e & 1]);
                        oq[e & 1] = fmaf(sd, qq[e], oq[e & 1]);
                        kq[e & 1] = fmaf(kk[e], qq[e], kq[e & 1]);
                    }
                }
                float p = pred[0] + pred[1], oqs = oq[0] + oq[1], kqs = kq[0] + kq[1];
#pragma unroll
                for (int off = 1; off < DG; off <<= 1) {
                    p += __shfl_xor_sync(0xffffffffu, p, off);
                    oqs += __shfl_xor_sync(0xffffffffu, oqs, off);
                    kqs += __shfl_xor_sync(0xffffffffu, kqs, off);
                }
                const float u = beta * (vj - p);
#pragma unroll
                for (int i4 = 0; i4 < NS / 4; ++i4) {
                    const float4 k4 = *reinterpret_cast<const float4*>(&s_k[buf][tt][(i4 * DG + dg) * 4]);
                    S[4 * i4 + 0] = fmaf(k4.x, u, S[4 * i4 + 0]);
                    S[4 * i4 + 1] = fmaf(k4.y, u, S[4 * i4 + 1]);
                    S[4 * i4 + 2] = fmaf(k4.z, u, S[4 * i4 + 2]);
                    S[4 * i4 + 3] = fmaf(k4.w, u, S[4 * i4 + 3]);
                }
                o = fmaf(u, kqs, oqs);
            } else {
                float ro[2] = {0.0f, 0.0f}, ruk[2] = {0.0f, 0.0f};
#pragma unroll
                for (int i4 = 0; i4 < NS / 4; ++i4) {
                    const int d = (i4 * DG + dg) * 4;
                    const float4 g4 = *reinterpret_cast<const float4*>(&s_g[buf][tt][HEAD ? 0 : d]);
                    const float4 k4 = *reinterpret_cast<const float4*>(&s_k[buf][tt][d]);
                    const float4 q4 = *reinterpret_cast<const float4*>(&s_q[buf][tt][d]);
                    const float gg[4] = {g4.x, g4.y, g4.z, g4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        ro[e & 1] = fmaf(qq[e], S[4 * i4 + e], ro[e & 1]);
                        ruk[e & 1] = fmaf(qq[e] * bonus[4 * i4 + e], kk[e], ruk[e & 1]);
                        S[4 * i4 + e] = fmaf(gg[e], S[4 * i4 + e], kk[e] * vj);
                    }
                }
                float rs = ro[0] + ro[1], us = ruk[0] + ruk[1];
#pragma unroll
                for (int off = 1; off < DG; off <<= 1) {
                    rs += __shfl_xor_sync(0xffffffffu, rs, off);
                    us += __shfl_xor_sync(0xffffffffu, us, off);
                }
                o = fmaf(vj, us, rs);
            }
            if (dg == 0 && col_ok) orow[(size_t)(base + tt) * ((size_t)a.heads * Dv)] = o;
        }
        __syncthreads();
    }
    if (col_ok) {
#pragma unroll
        for (int i = 0; i < NS; ++i) {
            const int d = ((i >> 2) * DG + dg) * 4 + (i & 3);
            if (d < D) sbase[(size_t)d * Dv] = S[i];
        }
    }
    rs_move_tail(a, slot, t0, n);
}

// ------------------------------------------------------------------------------------------ chunks of eight tokens
// The delta rule with one decay per head, eight tokens at a time.  With S0 the state ahead of a chunk, G_i = g_0 .. g_i and
// L_ij = g_(j+1) .. g_i, unrolling the recurrence gives
//     u_i + beta_i sum_{j<i} L_ij (k_i . k_j) u_j = beta_i (v_i - G_i S0^T k_i)
//     o_i = G_i S0^T q_i + sum_{j<=i} L_ij (q_i . k_j) u_j
//     S   = G_7 S0 + sum_j L_7j k_j u_j
// The matrix on the left depends on keys, decays and betas alone: its inverse, times beta, is the same for every value
// column.  delta_chunk_coef_kernel works out, for all chunks of all requests at once, the rows of that inverse, of
// L_ij (q_i . k_j), G_i and L_7i (RS_COEF floats a token and head); delta_chunk_kernel then walks the chunks of a request.
// The sums over key channels (S0^T k_i, S0^T q_i) of the eight tokens do not wait for one another, so a chunk costs one
// chain of dot products, a few shuffles and one update of the state where eight tokens cost eight.  All float32.
#define RS_CHUNK 8
#define RS_COEF 20

// Sums of x[0..N-1] over groups of N lanes: lane l of the group ends with the sum of x[l], in x[0].
template <int N>
__device__ __forceinline__ void rs_scatter_sum(float (&x)[N], int lane) {
#pragma unroll
    for (int off = N / 2; off >= 1; off >>= 1) {
        const bool up = (lane & off) != 0;
#pragma unroll
        for (int j = 0; j < off; ++j) {
            const float send = up ? x[j] : x[j + off], keep = up ? x[j + off] : x[j];
            x[j] = keep + __shfl_xor_sync(0xffffffffu, send, off);
        }
    }
}

// One warp per (chunk, head); blockIdx.x counts the chunks of all requests.  coef [T][heads][RS_COEF].
template <int SL>      // D <= 32 * SL
__global__ __launch_bounds__(128) void delta_chunk_coef_kernel(RecurrentArgs a, int num_reqs, float* __restrict__ coef) {
    pdl_trigger();
    pdl_wait();
    __shared__ float s_dot[4][64], s_m[4][RS_CHUNK][RS_CHUNK];
    int b = blockIdx.x, row0 = -1, nt = 0;
    for (int r = 0; r < num_reqs; ++r) {
        const int t0 = a.cu_tokens[r], n = a.cu_tokens[r + 1] - t0;
        if (n <= 0) continue;
        const int chunks = (n + RS_CHUNK - 1) / RS_CHUNK;
        if (b < chunks) { row0 = t0 + b * RS_CHUNK; nt = min(RS_CHUNK, n - b * RS_CHUNK); break; }
        b -= chunks;
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y * 4 + warp;
    if (row0 < 0 || head >= a.heads) return;
    const float* qh = a.q + (size_t)(head / a.kv_rep) * a.D;
    const float* kh = a.k + (size_t)(head / a.kv_rep) * a.D;
    // the 28 products k_i . k_j (j < i), then the 36 products q_i . k_j (j <= i)
    float acc[64];
#pragma unroll
    for (int e = 0; e < 64; ++e) acc[e] = 0.0f;
#pragma unroll
    for (int sl = 0; sl < SL; ++sl) {
        const int d = lane + 32 * sl;
        float kk[RS_CHUNK], qq[RS_CHUNK];
#pragma unroll
        for (int i = 0; i < RS_CHUNK; ++i) {
            const bool on = i < nt && d < a.D;
            kk[i] = on ? kh[(size_t)(row0 + i) * a.k_stride + d] : 0.0f;
            qq[i] = on ? qh[(size_t)(row0 + i) * a.q_stride + d] : 0.0f;
        }
        int e = 0;
#pragma unroll
        for (int i = 0; i < RS_CHUNK; ++i)
#pragma unroll
            for (int j = 0; j < i; ++j) { acc[e] = fmaf(kk[i], kk[j], acc[e]); ++e; }
#pragma unroll
        for (int i = 0; i < RS_CHUNK; ++i)
#pragma unroll
            for (int j = 0; j <= i; ++j) { acc[e] = fmaf(qq[i], kk[j], acc[e]); ++e; }
    }
    float half[2][32];
    // 64 sums over 32 lanes: value 2l and 2l + 1 end in lane l
#pragma unroll
    for (int e = 0; e < 32; ++e) { half[0][e] = acc[2 * e]; half[1][e] = acc[2 * e + 1]; }
    rs_scatter_sum<32>(half[0], lane);
    rs_scatter_sum<32>(half[1], lane);
    s_dot[warp][2 * lane] = half[0][0];
    s_dot[warp][2 * lane + 1] = half[1][0];
    __syncwarp();
    const int c = lane & (RS_CHUNK - 1);                 // lanes 8.. repeat what lanes 0..7 do and store nothing
    float g = 1.0f, beta = 0.0f;
    if (c < nt) {
        const float z = a.g[(size_t)(row0 + c) * a.g_stride + head] + a.dt_bias[head];
        g = expf(-expf(a.a_log[head]) * (fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)))));
        beta = 1.0f / (1.0f + expf(-a.beta[(size_t)(row0 + c) * a.beta_stride + head]));
    }
    // column c of L_ij k_i . k_j and of L_ij q_i . k_j; the decays up to and after token c
    float qk[RS_CHUNK], before = 1.0f, after = 1.0f, L = 1.0f;
#pragma unroll
    for (int i = 0; i < RS_CHUNK; ++i) {
        const float gi = __shfl_sync(0xffffffffu, g, i);
        if (i <= c) before *= gi;
        if (i > c) { after *= gi; L *= gi; }
        qk[i] = i >= c ? L * s_dot[warp][28 + i * (i + 1) / 2 + c] : 0.0f;
        if (lane < RS_CHUNK) s_m[warp][i][c] = i > c ? L * s_dot[warp][i * (i - 1) / 2 + c] : 0.0f;
    }
    __syncwarp();
    // column c of (I + diag(beta) M)^-1 diag(beta) by forward substitution
    float x[RS_CHUNK];
#pragma unroll
    for (int i = 0; i < RS_CHUNK; ++i) {
        const float bi = __shfl_sync(0xffffffffu, beta, i);
        float sum = 0.0f;
#pragma unroll
        for (int j = 0; j < i; ++j) sum = fmaf(s_m[warp][i][j], x[j], sum);
        x[i] = i < c ? 0.0f : i == c ? bi : -bi * sum;
    }
    if (lane < RS_CHUNK) {
        float* dst = coef + ((size_t)row0 * a.heads + head) * RS_COEF;
        const size_t step = (size_t)a.heads * RS_COEF;
#pragma unroll
        for (int i = 0; i < RS_CHUNK; ++i)
            if (i < nt) { dst[i * step + c] = x[i]; dst[i * step + RS_CHUNK + c] = qk[i]; }
        if (c < nt) { dst[c * step + 2 * RS_CHUNK] = before; dst[c * step + 2 * RS_CHUNK + 1] = after; }
    }
}

// two float32 numbers in a register pair: d = a * b + c and a * b, both halves at once
typedef unsigned long long rs_pair;
__device__ __forceinline__ rs_pair rs_fma2(rs_pair a, rs_pair b, rs_pair c) {
    rs_pair d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ rs_pair rs_mul2(rs_pair a, rs_pair b) {
    rs_pair d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ rs_pair rs_pack(float lo, float hi) {
    rs_pair d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 rs_unpack(rs_pair v) {
    float2 d;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(v));
    return d;
}

// One block per (request, head, 16 value columns), 256 threads: a column is shared by sixteen neighbouring lanes with NS key
// channels each.  After the sums over key channels lane l < 8 of a column holds token l's prediction and stands for its
// write, lane l >= 8 holds token l - 8's read-out of the old state and stands for its output.  (What bounds a prompt is how
// long one chunk takes, with few warps an SM: sixteen lanes a column instead of eight are twice the warps for the same work.)
template <int NS>
__global__ __launch_bounds__(256, NS <= 8 ? 2 : 1) void delta_chunk_kernel(RecurrentArgs a, const float* __restrict__ coef) {
    pdl_trigger();
    pdl_wait();
    constexpr int DG = 16, DP = NS * DG, COLS = 16, TT = NS >= 16 ? 8 : 16, NT = 256;
    constexpr bool KEEP_K = NS <= 8;              // the keys of a chunk stay in registers from the dot products to the update
    __shared__ __align__(16) float s_q[2][TT][DP], s_k[2][TT][DP], s_v[2][TT][COLS], s_c[2][TT][RS_COEF];
    __shared__ __align__(16) float s_x[NT / 32][32 / DG][3][RS_CHUNK];        // per warp and column: what its lanes tell one another
    const int r = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * COLS;
    const int t0 = a.cu_tokens[r], n = a.cu_tokens[r + 1] - t0;
    if (n <= 0) return;
    const int slot = a.state_slots[r];
    if (slot < 0 || slot >= a.max_slots) {
        if (threadIdx.x == 0) atomicOr(a.err, AIRUN_DEV_BAD_REQ);
        return;
    }
    const int D = a.D, Dv = a.Dv;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int dg = lane & (DG - 1), tok = dg & (RS_CHUNK - 1), cl = warp * (32 / DG) + lane / DG, col = col0 + cl;
    const bool col_ok = col < Dv;
    const int ncol = min(COLS, Dv - col0);
    // both stages start as zeros: padding and rows beyond the last token hold numbers whose weight is zero
    for (int e = threadIdx.x; e < 2 * TT * DP; e += NT) { (&s_q[0][0][0])[e] = 0.0f; (&s_k[0][0][0])[e] = 0.0f; }
    for (int e = threadIdx.x; e < 2 * TT * COLS; e += NT) (&s_v[0][0][0])[e] = 0.0f;
    __syncthreads();
    const float* qh = a.q + (size_t)(head / a.kv_rep) * D + (size_t)t0 * a.q_stride;
    const float* kh = a.k + (size_t)(head / a.kv_rep) * D + (size_t)t0 * a.k_stride;
    const float* vh = a.v + (size_t)head * Dv + col0 + (size_t)t0 * a.v_stride;
    const float* ch = coef + ((size_t)t0 * a.heads + head) * RS_COEF;
    // A thread copies the same piece of a row, of every step-th row: 16 bytes, or one number where the rows allow no more.
    const bool vec = (D % 4 == 0) && ((a.q_stride | a.k_stride) % 4 == 0) && ((((uintptr_t)qh | (uintptr_t)kh) & 15) == 0);
    const bool vvec = (ncol % 4 == 0) && (a.v_stride % 4 == 0) && (((uintptr_t)vh & 15) == 0);
    const int dper = vec ? D / 4 : min(D, NT), drows = NT / dper, drow = threadIdx.x / dper, dcol = (threadIdx.x - drow * dper) * (vec ? 4 : 1);
    const int vper = vvec ? ncol / 4 : ncol, vrows = NT / vper, vrow = threadIdx.x / vper, vcol = (threadIdx.x - vrow * vper) * (vvec ? 4 : 1);
    constexpr int CPER = RS_COEF / 4, CROWS = NT / CPER;
    const int crow = threadIdx.x / CPER, ccol = (threadIdx.x - crow * CPER) * 4;
    auto stage = [&](int base, int buf) {
        const int nt = min(TT, n - base);
        if (drow < drows)
            for (int tt = drow; tt < nt; tt += drows) {
                const float* qr = qh + (size_t)(base + tt) * a.q_stride;
                const float* kr = kh + (size_t)(base + tt) * a.k_stride;
                if (vec) {
                    rs_cp16(&s_q[buf][tt][dcol], qr + dcol);
                    rs_cp16(&s_k[buf][tt][dcol], kr + dcol);
                } else {
                    for (int d = dcol; d < D; d += dper) { rs_cp4(&s_q[buf][tt][d], qr + d); rs_cp4(&s_k[buf][tt][d], kr + d); }
                }
            }
        if (vrow < vrows)
            for (int tt = vrow; tt < nt; tt += vrows) {
                if (vvec) rs_cp16(&s_v[buf][tt][vcol], vh + (size_t)(base + tt) * a.v_stride + vcol);
                else rs_cp4(&s_v[buf][tt][vcol], vh + (size_t)(base + tt) * a.v_stride + vcol);
            }
        if (crow < CROWS)
            for (int tt = crow; tt < TT; tt += CROWS) {
                if (tt < nt) rs_cp16(&s_c[buf][tt][ccol], ch + (size_t)(base + tt) * a.heads * RS_COEF + ccol);
                else *reinterpret_cast<float4*>(&s_c[buf][tt][ccol]) = make_float4(0.f, 0.f, 0.f, 0.f);
            }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    float* sbase = a.state + (size_t)slot * a.slot_stride + (size_t)head * D * Dv + (col_ok ? col : 0);
    rs_pair S[NS / 2];                            // channel of number i: group of four (i / 4) * DG + dg, element i % 4
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
        float v[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int d = (((2 * i + h) >> 2) * DG + dg) * 4 + ((2 * i + h) & 3);
            v[h] = (col_ok && d < D) ? sbase[(size_t)d * Dv] : 0.0f;
        }
        S[i] = rs_pack(v[0], v[1]);
    }
    float* orow = a.out + (size_t)t0 * ((size_t)a.heads * Dv) + (size_t)head * Dv + col;
    float (*sx)[RS_CHUNK] = s_x[warp][lane / DG];
    int it = 0;
    for (int base = 0; base < n; base += TT, ++it) {
        const int buf = it & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                      // this stage is there, and nobody reads the other one any more
        if (base + TT < n) stage(base + TT, buf ^ 1);
#pragma unroll 1
        for (int c0 = 0; c0 < TT && base + c0 < n; c0 += RS_CHUNK) {
            const int nt = min(RS_CHUNK, n - base - c0);
            rs_pair p2[RS_CHUNK], o2[RS_CHUNK];
            ulonglong2 kr[KEEP_K ? RS_CHUNK : 1][KEEP_K ? NS / 4 : 1];
#pragma unroll
            for (int i = 0; i < RS_CHUNK; ++i) { p2[i] = 0ull; o2[i] = 0ull; }
#pragma unroll
            for (int i4 = 0; i4 < NS / 4; ++i4) {
#pragma unroll
                for (int i = 0; i < RS_CHUNK; ++i) {
                    const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(&s_k[buf][c0 + i][(i4 * DG + dg) * 4]);
                    const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(&s_q[buf][c0 + i][(i4 * DG + dg) * 4]);
                    if (KEEP_K) kr[KEEP_K ? i : 0][KEEP_K ? i4 : 0] = k4;
                    p2[i] = rs_fma2(S[2 * i4], k4.x, p2[i]); o2[i] = rs_fma2(S[2 * i4], q4.x, o2[i]);
                    p2[i] = rs_fma2(S[2 * i4 + 1], k4.y, p2[i]); o2[i] = rs_fma2(S[2 * i4 + 1], q4.y, o2[i]);
                }
            }
            float sum[2 * RS_CHUNK];
#pragma unroll
            for (int i = 0; i < RS_CHUNK; ++i) {
                const float2 pv = rs_unpack(p2[i]), ov = rs_unpack(o2[i]);
                sum[i] = pv.x + pv.y; sum[RS_CHUNK + i] = ov.x + ov.y;
            }
            rs_scatter_sum<2 * RS_CHUNK>(sum, lane);
            // this lane's token from here on: c0 + tok; its row of the inverse (its write) or of the products (its output)
            const float* cf = &s_c[buf][c0 + tok][0];
            const float2 dec = *reinterpret_cast<const float2*>(cf + 16);         // decay up to the token; from after it to the chunk's end
            const ulonglong2 ra = *reinterpret_cast<const ulonglong2*>(cf + (dg & RS_CHUNK)), rb = *reinterpret_cast<const ulonglong2*>(cf + (dg & RS_CHUNK) + 4);
            if (dg < RS_CHUNK) sx[0][tok] = fmaf(-dec.x, sum[0], s_v[buf][c0 + tok][cl]);
            __syncwarp();
            auto row_times = [&](const float* v) {
                const ulonglong2 va = *reinterpret_cast<const ulonglong2*>(v), vb = *reinterpret_cast<const ulonglong2*>(v + 4);
                const float2 t = rs_unpack(rs_fma2(rb.y, vb.y, rs_fma2(rb.x, vb.x, rs_fma2(ra.y, va.y, rs_mul2(ra.x, va.x)))));
                return t.x + t.y;
            };
            const float u = row_times(sx[0]);
            if (dg < RS_CHUNK) { sx[1][tok] = u; sx[2][tok] = u * dec.y; }
            const float whole = s_c[buf][c0 + nt - 1][16];
            const rs_pair w2 = rs_pack(whole, whole);
#pragma unroll
            for (int i = 0; i < NS / 2; ++i) S[i] = rs_mul2(S[i], w2);
            __syncwarp();
            const float4 wa = *reinterpret_cast<const float4*>(&sx[2][0]), wb = *reinterpret_cast<const float4*>(&sx[2][4]);
            const float w[RS_CHUNK] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
#pragma unroll
            for (int j = 0; j < RS_CHUNK; ++j) {
                const rs_pair wj = rs_pack(w[j], w[j]);
#pragma unroll
                for (int i4 = 0; i4 < NS / 4; ++i4) {
                    const ulonglong2 k4 = KEEP_K ? kr[KEEP_K ? j : 0][KEEP_K ? i4 : 0]
                                                 : *reinterpret_cast<const ulonglong2*>(&s_k[buf][c0 + j][(i4 * DG + dg) * 4]);
                    S[2 * i4] = rs_fma2(k4.x, wj, S[2 * i4]);
                    S[2 * i4 + 1] = rs_fma2(k4.y, wj, S[2 * i4 + 1]);
                }
            }
            const float o = fmaf(dec.x, sum[0], row_times(sx[1]));
            if (col_ok && dg >= RS_CHUNK && tok < nt) orow[(size_t)(base + c0 + tok) * ((size_t)a.heads * Dv)] = o;
            __syncwarp();                                     // the lanes' numbers are read before the next chunk's are written
        }
    }
    if (col_ok) {
#pragma unroll
        for (int i = 0; i < NS / 2; ++i) {
            const float2 v = rs_unpack(S[i]);
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int d = (((2 * i + h) >> 2) * DG + dg) * 4 + ((2 * i + h) & 3);
                if (d < D) sbase[(size_t)d * Dv] = h ? v.y : v.x;
            }
        }
    }
    rs_move_tail(a, slot, t0, n);
}

// `coef` (delta with one decay per head; [T][heads][RS_COEF] floats, 16-byte aligned, may be null): chunks of eight tokens.
AIRUN_EXPORT int airun_recurrent_state(int mode, const float* q, const float* k, const float* v, const float* g,
                                       long long q_stride, long long k_stride, long long v_stride, long long g_stride,
                                       const float* beta, long long beta_stride, const float* a_log, const float* dt_bias,
                                       const float* bonus, float* state,
                                       long long slot_stride, int max_slots, const int32_t* cu_tokens, const int32_t* state_slots,
                                       int num_reqs, float* out, int heads, int kv_rep, int D, int Dv, const float* tail_src,
                                       long long tail_src_stride, long long tail_off, int tail_rows, int tail_width,
                                       int long_chains, float* coef, int T, int* err, cudaStream_t stream) {
    if (num_reqs < 0 || heads <= 0 || heads > 65535 || kv_rep <= 0 || heads % kv_rep || D <= 0 || D > 256 || Dv <= 0 || !state ||
        !cu_tokens || !state_slots || !err || !q || !k || !v || !g || !out || slot_stride < (long long)heads * D * Dv)
        return AIRUN_ERR_ARG;
    if (mode < RS_DELTA || mode > RS_DELTA_HEAD || (mode == RS_WKV ? !bonus : !beta) || (mode == RS_DELTA_HEAD && (!a_log || !dt_bias)))
        return AIRUN_ERR_ARG;
    if (tail_rows < 0 || (tail_rows > 0 && (!tail_src || tail_width <= 0))) return AIRUN_ERR_ARG;
    if (num_reqs == 0) return AIRUN_OK;
    // lanes that share a value column: 8 where requests bring many tokens (the chain of a prompt's tokens bounds the
    // step, and a warp's instructions per token halve), 4 where most bring one (the state is read and written once, in
    // wider pieces)
    const int dg = (D <= 32 || !long_chains) ? 4 : 8;
    const int tiles = ceil_div_i(Dv, 128 / dg);
    if (tiles > 65535) return AIRUN_ERR_ARG;
    RecurrentArgs a = {q, k, v, g, q_stride, k_stride, v_stride, g_stride, beta, beta_stride, a_log, dt_bias, bonus, state, slot_stride, max_slots,
                       cu_tokens, state_slots, out, heads, kv_rep, D, Dv, tail_src, tail_src_stride, tail_off, tail_rows,
                       tail_width, err};
    if (coef) {
        if (mode != RS_DELTA_HEAD || T <= 0 || ((uintptr_t)coef & 15)) return AIRUN_ERR_ARG;
        const dim3 cgrid(T / RS_CHUNK + num_reqs, ceil_div_i(heads, 4)), mgrid(num_reqs, heads, ceil_div_i(Dv, 16));
        if (mgrid.z > 65535) return AIRUN_ERR_ARG;
#define RS_COEFS(SL) airun_launch(delta_chunk_coef_kernel<SL>, cgrid, dim3(128), 0, stream, a, num_reqs, coef)
#define RS_CHUNKS(NS) airun_launch(delta_chunk_kernel<NS>, mgrid, dim3(256), 0, stream, a, (const float*)coef)
        if (D <= 32) RS_COEFS(1);
        else if (D <= 64) RS_COEFS(2);
        else if (D <= 128) RS_COEFS(4);
        else RS_COEFS(8);
        if (D <= 64) RS_CHUNKS(4);
        else if (D <= 128) RS_CHUNKS(8);
        else RS_CHUNKS(16);
#undef RS_COEFS
#undef RS_CHUNKS
        return airun_launch_status();
    }
    dim3 grid(num_reqs, heads, tiles);
#define RS_LAUNCH(NS, DG) \
    do { if (mode == RS_DELTA) airun_launch(recurrent_state_kernel<RS_DELTA, NS, DG>, grid, dim3(128), 0, stream, a); \
         else if (mode == RS_DELTA_HEAD) airun_launch(recurrent_state_kernel<RS_DELTA_HEAD, NS, DG>, grid, dim3(128), 0, stream, a); \
         else airun_launch(recurrent_state_kernel<RS_WKV, NS, DG>, grid, dim3(128), 0, stream, a); } while (0)
    if (D <= 16) RS_LAUNCH(4, 4);
    else if (D <= 32) RS_LAUNCH(8, 4);
    else if (D <= 64) { if (dg == 8) RS_LAUNCH(8, 8); else RS_LAUNCH(16, 4); }
    else if (D <= 128) { if (dg == 8) RS_LAUNCH(16, 8); else RS_LAUNCH(32, 4); }
    else { if (dg == 8) RS_LAUNCH(32, 8); else RS_LAUNCH(64, 4); }
#undef RS_LAUNCH
    return airun_launch_status();
}
