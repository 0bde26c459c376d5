// Attention over a cached latent on the tensor cores (mma.sync m16n8k16, bfloat16 operands, float32 sums).
//
// The formulas are those of latent_attention.cu: every cached row [c (R) | kr (rd)] is key AND value for all heads,
// s = scale * q_lat . row, a sliding window, a sink in the softmax's denominator, out = sum_j p_j c_j.  Because all
// heads share the rows, the rows of a product tile are (token, head) pairs: a CTA takes TOK consecutive tokens of
// one request times up to 16 * RW heads (RW row tiles of 16), reads every cached row the tokens see ONCE for all of
// them, and keeps 256 of the R output columns in registers (blockIdx.z picks the columns; the scores are computed
// again for every 256 columns, which is cheaper than a second trip of the probabilities through shared memory).
//
// 8 (or 4) warps = as many row tiles, key tiles of 32 rows, every warp takes all keys of a tile, tiles arrive by cp.async in
// two stages (the next one is on its way while this one is used).  Single decoded tokens have a kernel of their own below.
// Each head's result may be times a sigmoid (`gate`, see latent_attention.cu).
// A cached row is found through the request's block table.  A group of TOK batch rows that straddles two requests is handled
// request by request.  Every row keeps its own maximum and sum, so a token's result does not depend on the batch.
#include "common.cuh"

#define LM_CW 256                 // output columns of a CTA
#define LM_NT (LM_CW / 8)

__device__ __forceinline__ void lm_cp16(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
// ldmatrix on shared-memory addresses that are worked out once a tile and stepped by plain adds
__device__ __forceinline__ uint32_t lm_saddr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void lm_ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void lm_ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void lm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t lm_pack(float lo, float hi) {
    __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&h);
}

struct LatentMmaArgs {
    const __nv_bfloat16* qlat; __nv_bfloat16* out; const __nv_bfloat16* pool;
    const int32_t* block_table; int max_blocks;
    const int32_t* positions; const int32_t* req_of_token;
    int T, num_reqs, num_pages, page_size, H, R, rd, window;
    float scale_log2;             // scale * log2(e)
    const float* sink;
    const float* gate;            // [T][gate_stride]: head h's result is times sigmoid(gate[t][h]); null: no gate
    long long gate_stride;
    const int32_t* cu_tokens;     // where each request's rows begin, [num_reqs + 1]
    int skip_single;              // requests that bring ONE token are left to the kernel for single tokens
    float* partial;               // [splits][num_reqs][H * (R + 2)] (sums, then maximum and denominator per head): a single token's key slices
    int splits;
    int hg, tok;                  // heads of a CTA, tokens of a CTA
    int kd16, kdp;                // the row padded to k-steps of 16; the shared-memory row stride in elements
    int* err;
};

template <int RW>
__global__ __launch_bounds__(32 * RW, 1) void latent_attention_mma_kernel(LatentMmaArgs a) {
    pdl_trigger();
    pdl_wait();
    constexpr int NWARP = RW, NTHREAD = 32 * NWARP, STAGES = 2;
    constexpr int BN = 32;                       // cached rows of a tile
    constexpr int ROWS = 16 * RW;
    extern __shared__ __align__(16) uint8_t lm_smem[];
    __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(lm_smem);                  // [ROWS][kdp]
    __nv_bfloat16* s_k = s_q + (size_t)ROWS * a.kdp;                                 // [2][BN][kdp]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rw = warp;
    const int KD = a.R + a.rd, kdp = a.kdp;
    const int t0 = blockIdx.x * a.tok, t1 = min(t0 + a.tok, a.T);
    const int h0 = blockIdx.y * a.hg, c0 = blockIdx.z * LM_CW;
    const int g = lane >> 2, qd = lane & 3;
    const int chunks = KD / 8;                  // 16-byte pieces of a cached row

    for (int tb = t0; tb < t1;) {
        const int req = a.req_of_token[tb];
        int te = tb + 1;
        if (req < 0 || req >= a.num_reqs) {
            if (req >= a.num_reqs && threadIdx.x == 0) atomicOr(a.err, AIRUN_DEV_BAD_REQ);
            tb = te;
            continue;
        }
        while (te < t1 && a.req_of_token[te] == req) ++te;
        if (a.skip_single && a.cu_tokens[req + 1] - a.cu_tokens[req] == 1) {      // left to the kernel for single tokens
            tb = te;
            continue;
        }
        const int p_first = a.positions[tb], n_tok = te - tb;
        const int p_last = p_first + n_tok - 1;
        const int j_lo = a.window > 0 ? max(0, p_first - a.window + 1) : 0;
        const int tile0 = j_lo / BN, tile_end = p_last / BN + 1;
        const int32_t* bt = a.block_table + (size_t)req * a.max_blocks;
        __syncthreads();                         // the pass before is done with the shared memory
        // the padding behind a cached row's last element is zero in every stage; the tile loads never copy into it
        for (int e = threadIdx.x; e < STAGES * BN * (kdp / 8 - chunks); e += NTHREAD) {
            const int row = e / (kdp / 8 - chunks), ch = chunks + e - row * (kdp / 8 - chunks);
            *reinterpret_cast<uint4*>(s_k + (size_t)row * kdp + ch * 8) = make_uint4(0, 0, 0, 0);
        }
        // the queries: row r = (token r / hg, head h0 + r % hg); rows beyond the group and the padding are zero
        for (int r = warp; r < ROWS; r += NWARP) {            // a warp a row: what the row needs is worked out once
            const int tl = r / a.hg, h = h0 + r - tl * a.hg;
            const bool on = tl < n_tok && h < a.H;
            const __nv_bfloat16* src = a.qlat + ((size_t)(tb + (on ? tl : 0)) * a.H + (on ? h : 0)) * KD;
            for (int ch = lane; ch < kdp / 8; ch += 32) {
                uint4 v = make_uint4(0, 0, 0, 0);
                if (on && ch < chunks) v = *reinterpret_cast<const uint4*>(src + ch * 8);
                *reinterpret_cast<uint4*>(s_q + (size_t)r * kdp + ch * 8) = v;
            }
        }
        bool bad = false;
        auto load_tile = [&](int tile, int buf) {
            __nv_bfloat16* dst = s_k + (size_t)buf * BN * kdp;
            for (int kr = warp; kr < BN; kr += NWARP) {        // a warp a cached row: one page lookup for the whole row
                const int j = tile * BN + kr;
                const int blk = j / a.page_size;
                int page = -1;
                if (j <= p_last && j >= j_lo && blk < a.max_blocks) {
                    page = bt[blk];
                    if (page >= a.num_pages) { bad = true; page = -1; }
                }
                __nv_bfloat16* d = dst + (size_t)kr * kdp;
                if (page >= 0) {
                    const __nv_bfloat16* src = a.pool + ((size_t)page * a.page_size + (j - blk * a.page_size)) * KD;
                    for (int ch = lane; ch < chunks; ch += 32) lm_cp16(d + ch * 8, src + ch * 8);
                } else {
                    for (int ch = lane; ch < chunks; ch += 32) *reinterpret_cast<uint4*>(d + ch * 8) = make_uint4(0, 0, 0, 0);
                }
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        load_tile(tile0, 0);

        float o[LM_NT][4];
#pragma unroll
        for (int i = 0; i < LM_NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
        float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
        // the two rows of this thread: rw * 16 + g and + 8; their positions
        int pos_r[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int r = rw * 16 + g + 8 * i, tl = r / a.hg;
            pos_r[i] = (tl < n_tok && h0 + r - tl * a.hg < a.H) ? p_first + tl : -1;       // -1: the row sees nothing
        }
        const int n_pairs = min(LM_NT / 2, (a.R - c0 + 15) / 16);      // pairs of 8 output columns this CTA has

        for (int tile = tile0, it = 0; tile < tile_end; ++tile, ++it) {
            const int buf = it & 1;
            if (tile + 1 < tile_end) {
                load_tile(tile + 1, buf ^ 1);
                asm volatile("cp.async.wait_group 1;" ::: "memory");
            } else {
                asm volatile("cp.async.wait_group 0;" ::: "memory");
            }
            __syncthreads();
            const __nv_bfloat16* kt = s_k + (size_t)buf * BN * kdp;
            // S = Q K^T for this warp's 16 rows and the tile's cached rows
            float s[BN / 8][4];
#pragma unroll
            for (int i = 0; i < BN / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
            uint32_t qaddr = lm_saddr(s_q + (size_t)(rw * 16 + (lane & 15)) * kdp + (lane >> 4) * 8);
            uint32_t kaddr = lm_saddr(kt + (size_t)((lane & 7) + ((lane >> 4) << 3)) * kdp + ((lane >> 3) & 1) * 8);
            const uint32_t kstep = (uint32_t)(16 * kdp * 2);
#pragma unroll 4
            for (int k0 = 0; k0 < a.kd16; k0 += 16, qaddr += 32, kaddr += 32) {
                uint32_t af[4];
                lm_ldsm4(af, qaddr);
#pragma unroll
                for (int np = 0; np < BN / 16; ++np) {
                    uint32_t bf[4];
                    lm_ldsm4(bf, kaddr + np * kstep);
                    lm_mma(s[2 * np], af, bf[0], bf[1]);
                    lm_mma(s[2 * np + 1], af, bf[2], bf[3]);
                }
            }
            // scale, mask, online softmax (base 2)
            const int jbase = tile * BN + qd * 2;
            float tmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = e >> 1, j = jbase + nt * 8 + (e & 1);
                    const bool vis = j <= pos_r[i] && j >= j_lo && (a.window == 0 || pos_r[i] - j < a.window);
                    const float v = vis ? s[nt][e] * a.scale_log2 : -INFINITY;
                    s[nt][e] = v;
                    tmax[i] = fmaxf(tmax[i], v);
                }
            float corr[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 1));
                tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 2));
                const float m_new = fmaxf(m_run[i], tmax[i]);
                corr[i] = m_new == -INFINITY ? 1.0f : exp2f(m_run[i] - m_new);
                m_run[i] = m_new;
            }
            float psum[2] = {0.0f, 0.0f};
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = e >> 1;
                    const float p = m_run[i] == -INFINITY ? 0.0f : exp2f(s[nt][e] - m_run[i]);
                    s[nt][e] = p;
                    psum[i] += p;
                }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                psum[i] += __shfl_xor_sync(0xffffffffu, psum[i], 1);
                psum[i] += __shfl_xor_sync(0xffffffffu, psum[i], 2);
                l_run[i] = l_run[i] * corr[i] + psum[i];
            }
            if (corr[0] != 1.0f || corr[1] != 1.0f) {       // once the maxima have settled nothing is rescaled
#pragma unroll
                for (int i = 0; i < LM_NT; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
            }
            // O += P V, V = the first R elements of the same cached rows
            const uint32_t vaddr = lm_saddr(kt + (size_t)((lane & 7) + ((lane >> 3) & 1) * 8) * kdp + c0 + (lane >> 4) * 8);
#pragma unroll
            for (int ks = 0; ks < BN / 16; ++ks) {
                uint32_t pf[4] = {lm_pack(s[2 * ks][0], s[2 * ks][1]), lm_pack(s[2 * ks][2], s[2 * ks][3]),
                                  lm_pack(s[2 * ks + 1][0], s[2 * ks + 1][1]), lm_pack(s[2 * ks + 1][2], s[2 * ks + 1][3])};
#pragma unroll
                for (int np = 0; np < LM_NT / 2; ++np) {
                    if (np < n_pairs) {
                        uint32_t vf[4];
                        lm_ldsm4t(vf, vaddr + ks * kstep + np * 32);
                        lm_mma(o[2 * np], pf, vf[0], vf[1]);
                        lm_mma(o[2 * np + 1], pf, vf[2], vf[3]);
                    }
                }
            }
            __syncthreads();                     // everybody is done with this stage before it is loaded again
        }
        if (bad && lane == 0) atomicOr(a.err, AIRUN_DEV_BAD_PAGE);

#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int r = rw * 16 + g + 8 * i, tl = r / a.hg, h = h0 + r - tl * a.hg;
            if (tl >= n_tok || h >= a.H) continue;
            float m = m_run[i], l = l_run[i], scale_o = 1.0f;
            if (a.sink) {
                const float sk = a.sink[h] * 1.4426950408889634f;
                const float mf = fmaxf(m, sk);
                scale_o = m == -INFINITY ? 0.0f : exp2f(m - mf);
                l = l * scale_o + exp2f(sk - mf);
            }
            float inv = l > 0.0f ? scale_o / l : 0.0f;
            if (a.gate) inv /= 1.0f + __expf(-a.gate[(size_t)(tb + tl) * a.gate_stride + h]);
            __nv_bfloat16* dst = a.out + ((size_t)(tb + tl) * a.H + h) * a.R + c0;
#pragma unroll
            for (int nt = 0; nt < LM_NT; ++nt) {
                const int c = nt * 8 + qd * 2;
                if (c0 + c < a.R) dst[c] = __float2bfloat16_rn(o[nt][2 * i] * inv);
                if (c0 + c + 1 < a.R) dst[c + 1] = __float2bfloat16_rn(o[nt][2 * i + 1] * inv);
            }
        }
        tb = te;
    }
}

// ---------------------------------------------------------------------------------------------------------
// Single decoded tokens.  One CTA (8 warps) per (slice of the keys, group of 16 * RT heads, request that brings ONE token):
// the rows of the products are the heads, so a cached row is read once for all of them, and all R output columns stay in
// the CTA's registers.  Tiles of 64 cached rows arrive by cp.async in two stages.  In a tile
//   scores   warp w takes rows 16 (w % 4) .. + 15 and one half (w / 4) of the row's elements; the halves meet in shared memory
//   softmax  warp w takes 2 RT heads, all 64 scores of a head over its lanes, with the head's running maximum and sum
//   output   warp w takes the columns 16 (w + 8 i) .. + 15 over all 64 rows
// With one slice the result (sink, division, gate) goes to `out`; with several each slice writes its float32 sums, maximum
// and denominator to `partial` and latent_merge_kernel adds them up in slice order.
#define LG_KEYS 64
#define LG_SS (LG_KEYS + 8)       // row stride of the scores in shared memory
#define LG_PAIRS 5                // 16-column pieces of a warp: R <= 8 * 5 * 16
#define LG_LOG2E 1.4426950408889634f

template <int RT>
__global__ __launch_bounds__(256, 1) void latent_attention_group_kernel(LatentMmaArgs a) {
    pdl_trigger();
    pdl_wait();
    constexpr int ROWS = 16 * RT, RPW = ROWS / 8;
    extern __shared__ __align__(16) uint8_t lm_smem[];
    const int kdp = a.kdp, KD = a.R + a.rd, chunks = KD / 8;
    __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(lm_smem);                  // [ROWS][kdp]
    __nv_bfloat16* s_k = s_q + (size_t)ROWS * kdp;                                   // [2][64][kdp]
    float* s_s = reinterpret_cast<float*>(s_k + (size_t)2 * LG_KEYS * kdp);          // [2][ROWS][LG_SS]: the halves' scores
    __nv_bfloat16* s_p = reinterpret_cast<__nv_bfloat16*>(s_s + 2 * ROWS * LG_SS);   // [ROWS][LG_SS]: the weights
    float* s_c = reinterpret_cast<float*>(s_p + ROWS * LG_SS);                       // [ROWS] factors, then [ROWS] maxima and [ROWS] sums
    float* s_m = s_c + ROWS;
    float* s_l = s_m + ROWS;
    const int slice = blockIdx.x, h0 = blockIdx.y * ROWS, r = blockIdx.z;
    const int tok = a.cu_tokens[r];
    if (a.cu_tokens[r + 1] - tok != 1) return;
    const int pos = a.positions[tok];                      // the last key the token sees
    if (pos < 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, qd = lane & 3;
    const int first_key = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const int tiles = (pos - first_key) / LG_KEYS + 1, per_slice = (tiles + a.splits - 1) / a.splits;
    const int lo = first_key + slice * per_slice * LG_KEYS;
    const int hi = min(pos, first_key + (slice + 1) * per_slice * LG_KEYS - 1);
    const int32_t* bt = a.block_table + (size_t)r * a.max_blocks;
    // the queries; heads beyond the last one and the padding behind the rows are zero, in the stages too
    for (int row = warp; row < ROWS; row += 8) {
        const bool on = h0 + row < a.H;
        const __nv_bfloat16* src = a.qlat + ((size_t)tok * a.H + (on ? h0 + row : 0)) * KD;
        for (int ch = lane; ch < kdp / 8; ch += 32) {
            uint4 v = make_uint4(0, 0, 0, 0);
            if (on && ch < chunks) v = *reinterpret_cast<const uint4*>(src + ch * 8);
            *reinterpret_cast<uint4*>(s_q + (size_t)row * kdp + ch * 8) = v;
        }
    }
    for (int e = threadIdx.x; e < 2 * LG_KEYS * (kdp / 8 - chunks); e += 256) {
        const int row = e / (kdp / 8 - chunks), ch = chunks + e - row * (kdp / 8 - chunks);
        *reinterpret_cast<uint4*>(s_k + (size_t)row * kdp + ch * 8) = make_uint4(0, 0, 0, 0);
    }
    bool bad = false;
    auto load_tile = [&](int kbase, int buf) {             // warp w copies rows w, w + 8, ...; rows beyond the slice are zeros
        __nv_bfloat16* dst = s_k + (size_t)buf * LG_KEYS * kdp;
        int page[LG_KEYS / 8];
#pragma unroll
        for (int i = 0; i < LG_KEYS / 8; ++i) {            // the page lookups first, so that they are under way together
            const int j = kbase + warp + 8 * i, blk = j / a.page_size;
            page[i] = j <= hi && blk < a.max_blocks ? bt[blk] : (j <= hi ? -1 : -2);
        }
#pragma unroll
        for (int i = 0; i < LG_KEYS / 8; ++i) {
            const int row = warp + 8 * i, j = kbase + row;
            __nv_bfloat16* d = dst + (size_t)row * kdp;
            if (page[i] >= 0 && page[i] < a.num_pages) {
                const __nv_bfloat16* src = a.pool + ((size_t)page[i] * a.page_size + j % a.page_size) * KD;
                for (int ch = lane; ch < chunks; ch += 32) lm_cp16(d + ch * 8, src + ch * 8);
            } else {
                if (page[i] != -2) bad = true;
                for (int ch = lane; ch < chunks; ch += 32) *reinterpret_cast<uint4*>(d + ch * 8) = make_uint4(0, 0, 0, 0);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float o[RT][LG_PAIRS][8];
#pragma unroll
    for (int t = 0; t < RT; ++t)
#pragma unroll
        for (int i = 0; i < LG_PAIRS; ++i)
#pragma unroll
            for (int e = 0; e < 8; ++e) o[t][i][e] = 0.0f;
    float m_run[RPW], l_run[RPW];                          // of this warp's heads in the softmax, the same in all lanes
#pragma unroll
    for (int i = 0; i < RPW; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.0f; }
    const int kg = warp & 3, kh = warp >> 2;
    const int steps = a.kd16 / 16, half = (steps + 1) / 2;
    const int s0 = kh ? half : 0, s1 = kh ? steps : half;  // this warp's k-steps of a row
    const int pairs = (a.R + 15) / 16;

    if (lo <= hi) load_tile(lo, 0);
    int it = 0;
    for (int kbase = lo; kbase <= hi; kbase += LG_KEYS, ++it) {
        const int buf = it & 1;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                   // the tile is here, and everybody is done with the one before
        if (kbase + LG_KEYS <= hi) load_tile(kbase + LG_KEYS, buf ^ 1);
        const __nv_bfloat16* kt = s_k + (size_t)buf * LG_KEYS * kdp;
        {
            float s[RT][2][4];
#pragma unroll
            for (int t = 0; t < RT; ++t)
#pragma unroll
                for (int i = 0; i < 2; ++i) s[t][i][0] = s[t][i][1] = s[t][i][2] = s[t][i][3] = 0.0f;
            uint32_t qaddr = lm_saddr(s_q + (size_t)(lane & 15) * kdp + (lane >> 4) * 8 + s0 * 16);
            uint32_t kaddr = lm_saddr(kt + (size_t)(16 * kg + (lane & 7) + ((lane >> 4) << 3)) * kdp + ((lane >> 3) & 1) * 8 + s0 * 16);
            const uint32_t qstep = (uint32_t)(16 * kdp * 2);
#pragma unroll 4
            for (int st = s0; st < s1; ++st, qaddr += 32, kaddr += 32) {
                uint32_t bf[4];
                lm_ldsm4(bf, kaddr);
#pragma unroll
                for (int t = 0; t < RT; ++t) {
                    uint32_t af[4];
                    lm_ldsm4(af, qaddr + t * qstep);
                    lm_mma(s[t][0], af, bf[0], bf[1]);
                    lm_mma(s[t][1], af, bf[2], bf[3]);
                }
            }
            float* dst = s_s + (size_t)kh * ROWS * LG_SS + 16 * kg + 2 * qd;
#pragma unroll
            for (int t = 0; t < RT; ++t)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    *reinterpret_cast<float2*>(dst + (size_t)(16 * t + g) * LG_SS + 8 * i) = make_float2(s[t][i][0], s[t][i][1]);
                    *reinterpret_cast<float2*>(dst + (size_t)(16 * t + g + 8) * LG_SS + 8 * i) = make_float2(s[t][i][2], s[t][i][3]);
                }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
            const int row = warp * RPW + i;
            const float2 x0 = *reinterpret_cast<const float2*>(s_s + (size_t)row * LG_SS + 2 * lane);
            const float2 x1 = *reinterpret_cast<const float2*>(s_s + (size_t)(ROWS + row) * LG_SS + 2 * lane);
            const int j = kbase + 2 * lane;
            const float v0 = j <= hi ? (x0.x + x1.x) * a.scale_log2 : -INFINITY, v1 = j + 1 <= hi ? (x0.y + x1.y) * a.scale_log2 : -INFINITY;
            const float m_new = fmaxf(m_run[i], warp_max(fmaxf(v0, v1)));
            const float corr = m_new == -INFINITY ? 1.0f : exp2f(m_run[i] - m_new);
            const float p0 = m_new == -INFINITY ? 0.0f : exp2f(v0 - m_new), p1 = m_new == -INFINITY ? 0.0f : exp2f(v1 - m_new);
            m_run[i] = m_new;
            l_run[i] = l_run[i] * corr + warp_sum(p0 + p1);
            *reinterpret_cast<uint32_t*>(s_p + (size_t)row * LG_SS + 2 * lane) = lm_pack(p0, p1);
            if (lane == 0) s_c[row] = corr;
        }
        __syncthreads();
        const uint32_t vaddr = lm_saddr(kt + (size_t)((lane & 7) + ((lane >> 3) & 1) * 8) * kdp + (lane >> 4) * 8 + warp * 16);
        const uint32_t paddr = lm_saddr(s_p + (size_t)(lane & 15) * LG_SS + (lane >> 4) * 8);
        const uint32_t vstep = (uint32_t)(16 * kdp * 2);
#pragma unroll
        for (int t = 0; t < RT; ++t) {
            const float c0 = s_c[16 * t + g], c1 = s_c[16 * t + g + 8];
            if (c0 != 1.0f || c1 != 1.0f) {                // once the maxima have settled nothing is rescaled
#pragma unroll
                for (int i = 0; i < LG_PAIRS; ++i) {
                    o[t][i][0] *= c0; o[t][i][1] *= c0; o[t][i][2] *= c1; o[t][i][3] *= c1;
                    o[t][i][4] *= c0; o[t][i][5] *= c0; o[t][i][6] *= c1; o[t][i][7] *= c1;
                }
            }
        }
#pragma unroll
        for (int ks = 0; ks < LG_KEYS / 16; ++ks) {
            uint32_t pf[RT][4];
#pragma unroll
            for (int t = 0; t < RT; ++t) lm_ldsm4(pf[t], paddr + t * (uint32_t)(16 * LG_SS * 2) + ks * 32);
#pragma unroll
            for (int i = 0; i < LG_PAIRS; ++i) {
                if (warp + 8 * i < pairs) {
                    uint32_t vf[4];
                    lm_ldsm4t(vf, vaddr + ks * vstep + i * 256);
#pragma unroll
                    for (int t = 0; t < RT; ++t) {
                        lm_mma(*reinterpret_cast<float(*)[4]>(&o[t][i][0]), pf[t], vf[0], vf[1]);
                        lm_mma(*reinterpret_cast<float(*)[4]>(&o[t][i][4]), pf[t], vf[2], vf[3]);
                    }
                }
            }
        }
    }
    if (bad && lane == 0) atomicOr(a.err, AIRUN_DEV_BAD_PAGE);
#pragma unroll
    for (int i = 0; i < RPW; ++i)
        if (lane == 0) { s_m[warp * RPW + i] = m_run[i]; s_l[warp * RPW + i] = l_run[i]; }
    __syncthreads();
#pragma unroll
    for (int t = 0; t < RT; ++t)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int row = 16 * t + g + 8 * u, h = h0 + row;
            if (h >= a.H) continue;
            const float m = s_m[row], l = s_l[row];
            if (a.splits > 1) {
                float* base = a.partial + ((size_t)slice * a.num_reqs + r) * ((size_t)a.H * (a.R + 2));
                float* dst = base + (size_t)h * a.R;
#pragma unroll
                for (int i = 0; i < LG_PAIRS; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int c = (warp + 8 * i) * 16 + (e >> 1) * 8 + 2 * qd + (e & 1);
                        if (c < a.R) dst[c] = o[t][i][(e >> 1) * 4 + 2 * u + (e & 1)];
                    }
                if (warp == 0 && qd == 0) {
                    base[(size_t)a.H * a.R + 2 * h] = m;
                    base[(size_t)a.H * a.R + 2 * h + 1] = l;
                }
                continue;
            }
            const float sk = a.sink ? a.sink[h] * LG_LOG2E : -INFINITY, top = fmaxf(m, sk);
            const float f = m == -INFINITY ? 0.0f : exp2f(m - top);
            const float den = l * f + (a.sink ? exp2f(sk - top) : 0.0f);
            float inv = den > 0.0f ? f / den : 0.0f;
            if (a.gate) inv /= 1.0f + __expf(-a.gate[(size_t)tok * a.gate_stride + h]);
            __nv_bfloat16* dst = a.out + ((size_t)tok * a.H + h) * a.R;
#pragma unroll
            for (int i = 0; i < LG_PAIRS; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int c = (warp + 8 * i) * 16 + (e >> 1) * 8 + 2 * qd + (e & 1);
                    if (c < a.R) dst[c] = __float2bfloat16_rn(o[t][i][(e >> 1) * 4 + 2 * u + (e & 1)] * inv);
                }
        }
}

// The slices of every single token merged in slice order, with the sink and the gate.  One block per (request, head); lane
// s of every warp holds slice s's maximum and sum (at most 32 slices).
__global__ __launch_bounds__(128) void latent_merge_kernel(LatentMmaArgs a) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, h = blockIdx.y;
    const int tok = a.cu_tokens[r];
    if (a.cu_tokens[r + 1] - tok != 1) return;
    const int lane = threadIdx.x & 31;
    const size_t width = (size_t)a.H * (a.R + 2), slice = (size_t)a.num_reqs * width;
    const float* base = a.partial + (size_t)r * width;
    const float* ml = base + (size_t)a.H * a.R + 2 * h;
    const float m = lane < a.splits ? ml[lane * slice] : -INFINITY, l = lane < a.splits ? ml[lane * slice + 1] : 0.0f;
    const float sk = a.sink ? a.sink[h] * LG_LOG2E : -INFINITY;
    const float top = fmaxf(warp_max(m), sk);
    const float w = m == -INFINITY ? 0.0f : exp2f(m - top);
    const float den = warp_sum(l * w) + (a.sink ? exp2f(sk - top) : 0.0f);
    float inv = den > 0.0f ? 1.0f / den : 0.0f;
    if (a.gate) inv /= 1.0f + __expf(-a.gate[(size_t)tok * a.gate_stride + h]);
    const float* col = base + (size_t)h * a.R;
    __nv_bfloat16* dst = a.out + ((size_t)tok * a.H + h) * a.R;
    for (int c0 = 0; c0 < a.R; c0 += 128) {                // (every lane takes part in the shuffles)
        const int c = min(c0 + (int)threadIdx.x, a.R - 1);
        float acc = 0.0f;
#pragma unroll 4
        for (int s = 0; s < a.splits; ++s) acc = fmaf(col[s * slice + c], __shfl_sync(0xffffffffu, w, s), acc);
        if (c0 + (int)threadIdx.x < a.R) dst[c] = __float2bfloat16_rn(acc * inv);
    }
}

static bool lm_fill(LatentMmaArgs& a, const void* qlat, void* out, const void* pool, const int32_t* block_table, int max_blocks,
                    const int32_t* cu_tokens, const int32_t* positions, int T, int num_reqs, int num_pages, int page_size, int H, int R,
                    int rd, float scale, int window, const float* sink, const float* gate, long long gate_stride, int* err) {
    const int KD = R + rd;
    if (T < 0 || num_reqs < 0 || H <= 0 || R <= 0 || rd < 0 || KD % 8 != 0 || KD > 640 || page_size <= 0 || num_pages <= 0 ||
        max_blocks <= 0 || window < 0 || !err || !cu_tokens || !positions || (gate && gate_stride < H) ||
        (((uintptr_t)qlat | (uintptr_t)pool) & 15))
        return false;
    a.qlat = (const __nv_bfloat16*)qlat; a.out = (__nv_bfloat16*)out; a.pool = (const __nv_bfloat16*)pool;
    a.block_table = block_table; a.max_blocks = max_blocks; a.cu_tokens = cu_tokens; a.positions = positions;
    a.T = T; a.num_reqs = num_reqs; a.num_pages = num_pages; a.page_size = page_size; a.H = H; a.R = R; a.rd = rd; a.window = window;
    a.scale_log2 = scale * LG_LOG2E;
    a.sink = sink; a.gate = gate; a.gate_stride = gate_stride; a.err = err;
    a.kd16 = (KD + 15) / 16 * 16;
    a.kdp = a.kd16 + 8;
    a.splits = 1;
    return true;
}

// Prompt portions (and, with skip_single == 0, single tokens too).  qlat [T][H][R + rd], out [T][H][R], pool pages of
// [page_size][R + rd], all bfloat16.  Needs (R + rd) % 8 == 0 and rows of up to 640 elements.
AIRUN_EXPORT int airun_latent_attention_mma(const void* qlat, void* out, const void* pool, const int32_t* block_table,
                                            int max_blocks, const int32_t* cu_tokens, const int32_t* positions,
                                            const int32_t* req_of_token, int T, int num_reqs, int num_pages,
                                            int page_size, int H, int R, int rd, float scale, int window, const float* sink,
                                            const float* gate, long long gate_stride, int skip_single, int* err, cudaStream_t stream) {
    LatentMmaArgs a = {};
    if (!req_of_token || !lm_fill(a, qlat, out, pool, block_table, max_blocks, cu_tokens, positions, T, num_reqs, num_pages,
                                                page_size, H, R, rd, scale, window, sink, gate, gate_stride, err))
        return AIRUN_ERR_ARG;
    if (T == 0) return AIRUN_OK;
    a.req_of_token = req_of_token; a.skip_single = skip_single;
    // 8 row tiles (128 rows) a CTA when its queries and two key tiles fit the shared memory, else 4
    const size_t limit = 227 * 1024;
    const int rw = ((size_t)128 + 2 * 32) * a.kdp * 2 > limit ? 4 : 8, rows = 16 * rw;
    a.hg = H < rows ? H : rows;
    a.tok = rows / a.hg;
    const size_t smem = ((size_t)rows + 2 * 32) * a.kdp * 2;
    if (smem > limit) return AIRUN_ERR_ARG;
    dim3 grid(ceil_div_i(T, a.tok), ceil_div_i(H, a.hg), ceil_div_i(R, LM_CW));
    if (grid.y > 65535 || grid.z > 65535) return AIRUN_ERR_ARG;
    static unsigned long long conf4 = 0, conf8 = 0;
#define LM_LAUNCH(RW_, CONF) do { \
        auto kern = latent_attention_mma_kernel<RW_>; \
        if (first_on_device(CONF)) { \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit); \
            if (e != cudaSuccess) return (int)e; \
        } \
        airun_launch(kern, grid, dim3(32 * RW_), smem, stream, a); } while (0)
    if (rw == 8) LM_LAUNCH(8, conf8);
    else LM_LAUNCH(4, conf4);
#undef LM_LAUNCH
    return airun_launch_status();
}

// The single tokens of the batch (requests that bring one).  splits > 1: the keys of a token are cut into that many slices,
// and `partial` holds splits * num_reqs * H * (R + 2) floats.
AIRUN_EXPORT int airun_latent_attention_group(const void* qlat, void* out, const void* pool, const int32_t* block_table, int max_blocks,
                                              const int32_t* cu_tokens, const int32_t* positions, int T, int num_reqs, int num_pages,
                                              int page_size, int H, int R, int rd, float scale, int window, const float* sink,
                                              const float* gate, long long gate_stride, int splits, float* partial, int* err,
                                              cudaStream_t stream) {
    LatentMmaArgs a = {};
    if (!lm_fill(a, qlat, out, pool, block_table, max_blocks, cu_tokens, positions, T, num_reqs, num_pages, page_size, H, R, rd, scale,
                 window, sink, gate, gate_stride, err) ||
        splits < 1 || splits > 32 || (splits > 1 && !partial) || num_reqs > 65535 || H > 65535)
        return AIRUN_ERR_ARG;
    if (T == 0 || num_reqs == 0) return AIRUN_OK;
    a.splits = splits; a.partial = partial;
    const int rt = H > 16 ? 2 : 1, rows = 16 * rt;
    const size_t smem = ((size_t)rows + 2 * LG_KEYS) * a.kdp * 2 + (size_t)rows * LG_SS * (2 * 4 + 2) + (size_t)3 * rows * 4;
    const size_t limit = 227 * 1024;
    if (smem > limit) return AIRUN_ERR_ARG;
    dim3 grid(splits, ceil_div_i(H, rows), num_reqs);
    static unsigned long long conf1 = 0, conf2 = 0;
#define LG_LAUNCH(RT_, CONF) do { \
        auto kern = latent_attention_group_kernel<RT_>; \
        if (first_on_device(CONF)) { \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit); \
            if (e != cudaSuccess) return (int)e; \
        } \
        airun_launch(kern, grid, dim3(256), smem, stream, a); } while (0)
    if (rt == 2) LG_LAUNCH(2, conf2);
    else LG_LAUNCH(1, conf1);
#undef LG_LAUNCH
    int rc = airun_launch_status();
    if (rc != AIRUN_OK || splits == 1) return rc;
    airun_launch(latent_merge_kernel, dim3(num_reqs, H), dim3(128), 0, stream, a);
    return airun_launch_status();
}
