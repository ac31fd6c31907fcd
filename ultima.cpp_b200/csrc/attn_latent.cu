// Latent attention on the fifth-generation tensor cores: any number of query heads (up to 128) over ONE key head
// whose rows hold the values as their leading columns, for prompts and for decode steps, paged bfloat16 cache.
// Compiled for a number of 64-column blocks a key row takes (-DROW_BLOCKS=1..9: rows of up to 576 numbers, of
// which up to 512 are values); the row's width and the values' are arguments.
//
// One CTA takes 128 rows, a row being (token, head), and walks over tiles of BN keys.  A tile of key rows is
// fetched ONCE (TMA, 128-byte swizzle) and serves both products:
//   S_b = Q K^T     tcgen05.mma, both operands from shared memory; two score buffers in tensor memory, so the
//                   next tile's scores are formed while this tile's are used
//   softmax         four warps, one thread a row: tcgen05.ld of the row's BN scores, mask, running maximum and
//                   sum in float32, probabilities rounded to bfloat16 and stored back over the scores
//   O += P V        P from tensor memory, V the leading columns of the same tile as the N-major operand
// Values of more than 256 columns are cut into parts of 256 (tensor memory holds scores and 256 output columns):
// a CTA takes one part and forms the scores anew.  A key tile's place in the ring is given back when the product
// with its values has been formed.  The maximum a row's exponentials refer to is raised only when the true one
// has grown by more than 2^8, as in attn_tcgen05.cu, whose roles of warps and order of issue this kernel shares:
// warp 0 TMA, warp 1 MMA and tensor-memory allocation, warps 2-5 softmax.  Rows the sequence has not reached are
// zeroed in shared memory before their product as values.  Every wait has a time limit and raises a flag.
//
// Decode (one new token a sequence): blockIdx.x is a slice of the key range; with several slices the CTA writes
// (reference maximum, sum, unnormalised output) for attn_latent_combine_kernel.  Key tiles of earlier pages are
// asked for before the kernel in front (which writes the newest row) has ended.
//
// A learned sink (float32, one a head) is one more term exp(sink) in the softmax's sum that brings no value.
#include "common.cuh"
#include "tc_common.cuh"

#ifndef ROW_BLOCKS
#define ROW_BLOCKS 4
#endif
static_assert(ROW_BLOCKS >= 1 && ROW_BLOCKS <= 9, "key rows of 64 to 576 numbers");

constexpr int RB = ROW_BLOCKS;
constexpr int BM = 128;                       // rows a CTA
constexpr int PAGE = 64;                      // positions a page
constexpr int BN = RB >= 8 ? 32 : 64;         // keys a tile
constexpr int Q_BYTES = RB * BM * 128;
constexpr int KV_BYTES = RB * BN * 128;
constexpr int STAGES = RB == 1 ? 6 : RB == 2 ? 4 : RB == 3 ? 6 : RB == 4 ? 4 : RB == 5 ? 3 : RB == 8 ? 3 : 2;
constexpr int SMEM_BYTES = Q_BYTES + STAGES * KV_BYTES + 1024 + 256;
static_assert(SMEM_BYTES <= 232448, "ring and queries outgrew shared memory");
constexpr int O_COL = 2 * BN;                 // tensor memory: S0 [0, BN) S1 [BN, 2 BN) O [2 BN, 2 BN + values of the part)
constexpr int PART = 256;                     // value columns a CTA takes
constexpr int MAX_PART = RB * 64 < PART ? RB * 64 : PART;
constexpr int TMEM_COLS = O_COL + MAX_PART <= 128 ? 128 : O_COL + MAX_PART <= 256 ? 256 : 512;
constexpr float RESCALE_STEP = 8.0f;          // log2 units the reference maximum may lag behind
constexpr int NTHREADS = 192;
constexpr int CTAS_PER_SM = (RB <= 2 && TMEM_COLS <= 256) ? 2 : 1;
constexpr float LOG2E = 1.4426950408889634f;

typedef __nv_bfloat16 bf16;

struct LatentParams {
    bf16* out; long long o_stride;            // [tokens, heads, values], row stride o_stride
    const int* seq_start; const int* seq_before; const int* table;
    int pages_per_seq, ring, nh, row, vals, window;
    float c;                                  // scale * log2(e)
    const float* sink;                        // [heads] or null
    int* error;
    float* part_o; float* part_ml; int n_slices;      // decode in several slices: [seq, head, slice, vals], [.., 2]
    int n_seqs, n_row_tiles, n_parts;
};

__host__ __device__ constexpr uint32_t idesc_bf16(int m, int n, int b_mn_major) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)b_mn_major << 16) | ((uint32_t)(n >> 3) << 17) |
           ((uint32_t)(m >> 4) << 24);
}
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint64_t pair_of(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void halves_of(uint64_t v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t fma_pair(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t add_pair(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float max3(float a, float b, float c) {
    float d;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
    return d;
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
          "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
// Key tile as the N-major B operand: rows of 128 bytes are keys, 8 keys a swizzle atom (1024 bytes), 64 columns a block
__device__ __forceinline__ uint64_t make_desc_mn(uint32_t smem_addr) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
    d |= (uint64_t)((BN * 128) >> 4) << 16;                // next 64 columns
    d |= (uint64_t)(1024 >> 4) << 32;                      // next 8 keys
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}

template <bool DECODE>
__global__ void __launch_bounds__(NTHREADS, CTAS_PER_SM)
attn_latent_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, LatentParams p) {
    extern __shared__ uint8_t smem_raw[];
    // prompts: numbered so that the blocks with the most keys to visit are handed out first, a row tile's parts side by side
    const int per_tile = p.n_seqs * p.n_parts;
    const int seq = DECODE ? blockIdx.y : (blockIdx.x % per_tile) / p.n_parts;
    const int part = DECODE ? blockIdx.z : blockIdx.x % p.n_parts;
    const int q0 = p.seq_start[seq], q_len = p.seq_start[seq + 1] - q0, before = p.seq_before[seq];
    const int G = p.nh;
    const int TPB = BM / G;                                // tokens a tile: TPB * G of the 128 rows are in use
    const int tok_first = DECODE ? 0 : (p.n_row_tiles - 1 - (int)(blockIdx.x / per_tile)) * TPB;
    if (tok_first >= q_len) return;                        // (a block that ends counts as one that has let its dependents go)
    const int v0 = part * PART;                            // this part's value columns: [v0, v0 + nv)
    const int nv = min(PART, p.vals - v0);
    const int vn = (nv + 15) & ~15;                        // the product's N

    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint8_t* q_s = smem;
    uint8_t* k_s = q_s + Q_BYTES;
    uint64_t* bars = (uint64_t*)(k_s + STAGES * KV_BYTES);
    uint64_t* q_full = bars;
    uint64_t* k_full = bars + 1;
    uint64_t* k_empty = k_full + STAGES;
    uint64_t* s_full = k_empty + STAGES;                   // [2]
    uint64_t* p_full = s_full + 2;                         // [2]
    uint64_t* pv_done = p_full + 2;                        // [2]
    uint32_t* tmem_slot = (uint32_t*)(pv_done + 2);
    volatile int* err = (volatile int*)(tmem_slot + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int last_pos = before + q_len - 1;
    const int tok_last = DECODE ? 0 : min(q_len - 1, tok_first + TPB - 1);
    const int pos_hi = before + tok_last;
    const int pos_lo = span_lo(before + tok_first, p.window);
    int t_lo = pos_lo / BN, n_tiles = pos_hi / BN - t_lo + 1;
    if (DECODE) {                                          // this CTA's slice of the tiles (may be empty)
        const int per = (n_tiles + p.n_slices - 1) / p.n_slices;
        const int first = min(n_tiles, (int)blockIdx.x * per);
        n_tiles = min(n_tiles - first, per);
        t_lo += first;
    }

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int s = 0; s < STAGES; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&s_full[b], 1); mbar_init(&p_full[b], 4); mbar_init(&pv_done[b], 1); }
        *err = 0;
        fence_barrier_init();
    }
    if (warp == 1) { tmem_alloc(tmem_slot, TMEM_COLS); tmem_relinquish(); }
    if (warp == 0 && lane == 0) { prefetch_tmap(&map_q); prefetch_tmap(&map_k); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    // dependents are let go only now that this block holds its tensor memory (see attn_tcgen05.cu)
    pdl_trigger();

    auto load_tile = [&](int j) {                          // one thread: key tile j into its stage of the ring
        const int s = j % STAGES;
        const int posn = (t_lo + j) * BN;
        const int page = p.table[(long long)seq * p.pages_per_seq + (posn % p.ring) / PAGE];
        const int row0 = page * PAGE + posn % PAGE;
        mbar_expect_tx(&k_full[s], KV_BYTES);
        for (int nb = 0; nb < RB; ++nb) tma_load_2d(k_s + s * KV_BYTES + nb * BN * 128, &map_k, &k_full[s], nb * 64, row0);
    };
    int early = 0;
    if (DECODE && warp == 0 && lane == 0) {
        // pages before the newest position's were written by earlier steps
        while (early < n_tiles && early < STAGES && (t_lo + early) * BN / PAGE < pos_hi / PAGE) { load_tile(early); ++early; }
    }
    pdl_wait();

    if (warp == 0) {
        // ---------------- TMA ----------------
        if (lane == 0) {
            if (n_tiles > 0) {
                mbar_expect_tx(q_full, RB * TPB * G * 128);
                for (int nb = 0; nb < RB; ++nb) tma_load_3d(q_s + nb * BM * 128, &map_q, q_full, nb * 64, 0, q0 + tok_first);
            }
            int armed = early;
            for (int j = early; j < n_tiles; ++j) {
                if (!mbar_wait(&k_empty[j % STAGES], (uint32_t)(((j / STAGES) & 1) ^ 1), err)) break;
                load_tile(j);
                armed = j + 1;
            }
            if (*err) {          // let the copies in flight land before the CTA's memory goes away
                const long long tstart = clock64();
                while (n_tiles > 0 && !mbar_try_wait(q_full, 0)) if (clock64() - tstart > WAIT_LIMIT_CYCLES / 8) break;
                for (int j = max(0, armed - STAGES); j < armed; ++j)
                    while (!mbar_try_wait(&k_full[j % STAGES], (j / STAGES) & 1)) if (clock64() - tstart > WAIT_LIMIT_CYCLES / 4) break;
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA ----------------
        if (lane == 0) {
            constexpr uint32_t idesc_qk = idesc_bf16(BM, BN, 0);
            const uint32_t idesc_pv = idesc_bf16(BM, vn, 1);
            const uint64_t q_desc = make_desc(smem_u32(q_s));
            const uint64_t k_desc = make_desc(smem_u32(k_s));
            const uint64_t v_desc = make_desc_mn(smem_u32(k_s + (v0 / 64) * BN * 128));
            const int k_steps = (p.row + 15) / 16;
            auto issue_qk = [&](int j) {
                const uint64_t kd = k_desc + (uint64_t)((j % STAGES) * (KV_BYTES >> 4));
                const uint32_t acc = tmem_base + (uint32_t)((j & 1) * BN);
#pragma unroll
                for (int ks = 0; ks < RB * 4; ++ks) {
                    if (ks >= k_steps) break;
                    const uint64_t da = q_desc + (uint64_t)(((ks / 4) * BM * 128 + (ks % 4) * 32) >> 4);
                    const uint64_t db = kd + (uint64_t)(((ks / 4) * BN * 128 + (ks % 4) * 32) >> 4);
                    tc_mma_bf16(acc, da, db, idesc_qk, ks > 0 ? 1u : 0u);
                }
                tc_commit(&s_full[j & 1]);
            };
            // MMAs run in the order of their issue: the scores of tile j+1 may be queued over the place of tile j-1's
            // probabilities as soon as the product that reads those has been issued
            bool ok = n_tiles > 0 ? mbar_wait(q_full, 0, err) : true;
            if (ok && n_tiles > 0) ok = mbar_wait(&k_full[0], 0, err);
            if (ok && n_tiles > 0) { tc_fence_after(); issue_qk(0); }
            for (int j = 0; j < n_tiles && ok; ++j) {
                if (j + 1 < n_tiles) {
                    ok = mbar_wait(&k_full[(j + 1) % STAGES], (uint32_t)(((j + 1) / STAGES) & 1), err);
                    if (!ok) break;
                    tc_fence_after();
                    issue_qk(j + 1);
                }
                ok = mbar_wait(&p_full[j & 1], (uint32_t)((j >> 1) & 1), err);
                if (!ok) break;
                tc_fence_after();
                const uint64_t vd = v_desc + (uint64_t)((j % STAGES) * (KV_BYTES >> 4));
                const uint32_t p_t = tmem_base + (uint32_t)((j & 1) * BN);
#pragma unroll
                for (int ks = 0; ks < BN / 16; ++ks)
                    tc_mma_bf16_ts(tmem_base + O_COL, p_t + ks * 8, vd + (uint64_t)((ks * 16 * 128) >> 4), idesc_pv,
                                   (j > 0 || ks > 0) ? 1u : 0u);
                tc_commit(&pv_done[j & 1]);
                tc_commit(&k_empty[j % STAGES]);
            }
        }
    } else {
        // ---------------- softmax: one thread a row ----------------
        const int q = warp & 3;
        const int r = q * 32 + lane;                       // row of the tile = lane of tensor memory
        const int tok = tok_first + r / G, head = r % G;
        const bool row_ok = r < TPB * G && tok < q_len;
        const int row_pos = before + tok;
        const uint32_t lane_addr = tmem_base + ((uint32_t)(q * 32) << 16);
        const int st = (warp - 2) * 32 + lane;             // 0..127 among the softmax threads
        const bool partial = DECODE && p.n_slices > 1;
        float m_ref = -INFINITY, l = 0.f;
        if (p.sink && !partial) { m_ref = p.sink[head] * LOG2E; l = 1.f; }        // (slices: the sink joins where they are merged)
        bool ok = true;
        for (int j = 0; j < n_tiles && ok; ++j) {
            const int b = j & 1;
            const int base = (t_lo + j) * BN;
            if (base + BN - 1 > last_pos) {
                // key rows past the sequence's end hold whatever the page held before: zeros as values (their scores are masked)
                ok = mbar_wait(&k_full[j % STAGES], (uint32_t)((j / STAGES) & 1), err);
                if (!ok) break;
                const int first = last_pos + 1 - base;     // first row to clear (>= 1: the tile holds a valid key)
                uint8_t* kt = k_s + (j % STAGES) * KV_BYTES;
                for (int i = st; i < (BN - first) * RB * 8; i += 128) {
                    const int row = first + i / (RB * 8), rest = i % (RB * 8);
                    *reinterpret_cast<uint4*>(kt + (rest / 8) * BN * 128 + row * 128 + (rest % 8) * 16) = make_uint4(0, 0, 0, 0);
                }
                fence_proxy_async();
            }
            ok = mbar_wait(&s_full[b], (uint32_t)((j >> 1) & 1), err);
            if (!ok) break;
            tc_fence_after();
            uint32_t raw[BN];
#pragma unroll
            for (int i = 0; i < BN; i += 32) tmem_ld32(lane_addr + (uint32_t)(b * BN + i), raw + i);
            tmem_ld_wait();
            // a tile that every row of the warp sees whole needs no mask
            const bool whole = row_ok && base + BN - 1 <= before + tok_first && p.window == 0;
            if (!__all_sync(0xffffffffu, whole)) {
                const int row_lo = span_lo(row_pos, p.window);
#pragma unroll
                for (int cI = 0; cI < BN; ++cI) {
                    const int kp = base + cI;
                    if (!(row_ok && kp <= row_pos && kp >= row_lo)) raw[cI] = __float_as_uint(-INFINITY);
                }
            }
            float mxs[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int cI = 0; cI < BN; cI += 8)
#pragma unroll
                for (int ch = 0; ch < 4; ++ch)
                    mxs[ch] = max3(mxs[ch], __uint_as_float(raw[cI + 2 * ch]), __uint_as_float(raw[cI + 2 * ch + 1]));
            float mx = fmaxf(fmaxf(mxs[0], mxs[1]), fmaxf(mxs[2], mxs[3]));
            mx *= p.c;                                      // c > 0: the maximum in exponent units
            const bool grow = mx > m_ref + RESCALE_STEP || (m_ref == -INFINITY && mx > -INFINITY);
            if (__any_sync(0xffffffffu, grow)) {
                const float m_new = grow ? mx : m_ref;
                const float f = (m_ref == -INFINITY || !grow) ? (grow ? 0.f : 1.f) : exp2f(m_ref - m_new);
                if (j > 0) {
                    ok = mbar_wait(&pv_done[(j - 1) & 1], (uint32_t)(((j - 1) >> 1) & 1), err);   // O is at rest
                    if (!ok) break;
                    tc_fence_after();
                    for (int cb = 0; cb < vn; cb += 16) {
                        uint32_t oo[16];
                        tmem_ld16(lane_addr + (uint32_t)(O_COL + cb), oo);
                        tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 16; ++i) oo[i] = __float_as_uint(__uint_as_float(oo[i]) * f);
                        tmem_st16(lane_addr + (uint32_t)(O_COL + cb), oo);
                    }
                    tmem_st_wait();
                }
                l *= f;
                m_ref = m_new;
            }
            const float mb = m_ref == -INFINITY ? 0.f : m_ref;
            uint32_t packed[BN / 2];
            const uint64_t c2 = pair_of(p.c, p.c), shift2 = pair_of(-mb, -mb);
            uint64_t sums[2] = {pair_of(0.f, 0.f), pair_of(0.f, 0.f)};
#pragma unroll
            for (int cI = 0; cI < BN; cI += 2) {
                float x0, x1;
                halves_of(fma_pair(pair_of(__uint_as_float(raw[cI]), __uint_as_float(raw[cI + 1])), c2, shift2), x0, x1);
                const float p0 = ex2(x0), p1 = ex2(x1);
                sums[(cI >> 1) & 1] = add_pair(sums[(cI >> 1) & 1], pair_of(p0, p1));
                __nv_bfloat162 pr = __floats2bfloat162_rn(p0, p1);
                packed[cI / 2] = *reinterpret_cast<uint32_t*>(&pr);
            }
            float s0, s1, s2, s3;
            halves_of(sums[0], s0, s1);
            halves_of(sums[1], s2, s3);
            l += (s0 + s1) + (s2 + s3);
            if constexpr (BN == 64) tmem_st32(lane_addr + (uint32_t)(b * BN), packed);
            else tmem_st16(lane_addr + (uint32_t)(b * BN), packed);
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[b]);         // one arrival a warp
        }
        if (ok && n_tiles > 0) ok = mbar_wait(&pv_done[(n_tiles - 1) & 1], (uint32_t)(((n_tiles - 1) >> 1) & 1), err);
        if (ok) {
            tc_fence_after();
            const float inv = partial ? 1.0f : (l > 0.f ? 1.0f / l : 0.f);
            bf16* dst = p.out + (long long)(q0 + tok) * p.o_stride + (long long)head * p.vals + v0;
            const long long pi = partial ? ((long long)seq * p.nh + head) * p.n_slices + blockIdx.x : 0;
            if (partial && row_ok && part == 0) { p.part_ml[pi * 2] = m_ref; p.part_ml[pi * 2 + 1] = l; }
            for (int cb = 0; cb < vn; cb += 16) {
                uint32_t oo[16];
                if (n_tiles > 0) {
                    tmem_ld16(lane_addr + (uint32_t)(O_COL + cb), oo);
                    tmem_ld_wait();
                } else {
#pragma unroll
                    for (int i = 0; i < 16; ++i) oo[i] = 0;
                }
                if (!row_ok) continue;
#pragma unroll
                for (int i = 0; i < 16; i += 8) {
                    if (cb + i >= nv) break;                // (value columns come in eights)
                    if (partial) {
                        float* po = p.part_o + pi * p.vals + v0 + cb + i;
                        *reinterpret_cast<uint4*>(po) = make_uint4(oo[i], oo[i + 1], oo[i + 2], oo[i + 3]);
                        *reinterpret_cast<uint4*>(po + 4) = make_uint4(oo[i + 4], oo[i + 5], oo[i + 6], oo[i + 7]);
                    } else {
                        float v[8];
#pragma unroll
                        for (int e = 0; e < 8; ++e) v[e] = __uint_as_float(oo[i + e]) * inv;
                        store_vec<bf16, 8>(dst + cb + i, v);
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, TMEM_COLS);
    }
    if (threadIdx.x == 0 && *err) atomicExch(p.error, 1);
}

// merge the slices of a decode step: grid (sequences * heads), four value columns a thread
__global__ void attn_latent_combine_kernel(LatentParams p) {
    pdl_trigger();
    pdl_wait();
    const int sh = blockIdx.x, d = threadIdx.x * 4;
    const int seq = sh / p.nh, head = sh % p.nh;
    const long long base = (long long)sh * p.n_slices;
    float mm = -INFINITY;
#pragma unroll 8
    for (int s = 0; s < p.n_slices; ++s) mm = fmaxf(mm, p.part_ml[(base + s) * 2]);
    const float sk = p.sink ? p.sink[head] * LOG2E : -INFINITY;
    mm = fmaxf(mm, sk);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    float ll = p.sink ? exp2f(sk - mm) : 0.f;
    if (d >= p.vals) return;
#pragma unroll 8
    for (int s = 0; s < p.n_slices; ++s) {
        const float ms = p.part_ml[(base + s) * 2];
        const float f = ms == -INFINITY ? 0.f : exp2f(ms - mm);        // (an empty slice has written zeros)
        ll = fmaf(f, p.part_ml[(base + s) * 2 + 1], ll);
        const float4 o = *reinterpret_cast<const float4*>(p.part_o + (base + s) * p.vals + d);
        acc.x = fmaf(f, o.x, acc.x); acc.y = fmaf(f, o.y, acc.y); acc.z = fmaf(f, o.z, acc.z); acc.w = fmaf(f, o.w, acc.w);
    }
    const float inv = 1.0f / ll;
    const float v[4] = {acc.x * inv, acc.y * inv, acc.z * inv, acc.w * inv};
    store_vec<bf16, 4>(p.out + (long long)p.seq_start[seq] * p.o_stride + (long long)head * p.vals + d, v);
}

UB_API int ub_attn_latent_row_blocks() { return RB; }

// tensor map of the queries [tokens, heads, row] (token stride q_stride elements), boxes of 64 x heads x floor(128 / heads)
UB_API int ub_attn_latent_map_q(void* out_map, const void* q, long long n_tokens, int nh, long long q_stride, int row) {
    EncodeTiledFn enc = tensor_map_encoder();
    if (!enc) return UB_ERR_UNSUPPORTED;
    if (((uintptr_t)q & 15) || (q_stride * 2) % 16 != 0 || row % 8 != 0 || row > RB * 64 || row <= (RB - 1) * 64 || nh < 1 || nh > BM ||
        n_tokens < 1) return UB_ERR_ARG;
    cuuint64_t dims[3] = {(cuuint64_t)row, (cuuint64_t)nh, (cuuint64_t)n_tokens};
    cuuint64_t strides[2] = {(cuuint64_t)row * 2, (cuuint64_t)q_stride * 2};
    cuuint32_t box[3] = {64, (cuuint32_t)nh, (cuuint32_t)(BM / nh)};
    cuuint32_t estr[3] = {1, 1, 1};
    CUresult r = enc((CUtensorMap*)out_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, (void*)q, dims, strides, box, estr,
                     CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                     CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : UB_ERR_ARG;
}
// tensor map of one run's key rows [pages, 1, 64, row], boxes of 64 columns x BN keys, zeros past the row's width
UB_API int ub_attn_latent_map_k(void* out_map, const void* cache, long long n_pages, int row) {
    EncodeTiledFn enc = tensor_map_encoder();
    if (!enc) return UB_ERR_UNSUPPORTED;
    if (((uintptr_t)cache & 15) || n_pages < 1 || row % 8 != 0 || row > RB * 64 || row <= (RB - 1) * 64) return UB_ERR_ARG;
    cuuint64_t dims[2] = {(cuuint64_t)row, (cuuint64_t)(n_pages * PAGE)};
    cuuint64_t strides[1] = {(cuuint64_t)row * 2};
    cuuint32_t box[2] = {64, (cuuint32_t)BN};
    cuuint32_t estr[2] = {1, 1};
    CUresult r = enc((CUtensorMap*)out_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void*)cache, dims, strides, box, estr,
                     CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                     CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : UB_ERR_ARG;
}

template <bool DECODE>
static int launch_latent(dim3 grid, const void* map_q, const void* map_k, const LatentParams& p, cudaStream_t st) {
    static bool attr_done = false;
    auto kern = attn_latent_kernel<DECODE>;
    if (!attr_done) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_BYTES);
        if (e != cudaSuccess) return (int)e;
        attr_done = true;
    }
    return (int)ub_launch_dependent(kern, grid, dim3(NTHREADS), (size_t)SMEM_BYTES, st, *(const CUtensorMap*)map_q,
                                    *(const CUtensorMap*)map_k, p);
}

// decode 0: prompts (any numbers of new tokens); 1: one new token a sequence, keys in n_slices slices (part_o: float32
// [n_seqs, nh, n_slices, vals], part_ml: [.., 2] when n_slices > 1).  vals: value columns, a multiple of 8, at most the row's.
UB_API int ub_attn_latent(int decode, const void* map_q, const void* map_k, void* out, long long o_stride, const int* seq_start,
                          const int* seq_before, const int* table, int pages_per_seq, int ring, int page, int n_seqs, int max_new,
                          int nh, int row, int vals, int window, float scale, const float* sink, int n_slices, float* part_o,
                          float* part_ml, int* error, cudaStream_t st) {
    if (n_seqs <= 0 || max_new <= 0) return 0;
    if (page != PAGE || ring % page != 0 || nh < 1 || nh > BM || row > RB * 64 || row <= (RB - 1) * 64 || row % 8 != 0 || vals % 8 != 0 ||
        vals < 8 || vals > row || vals > 2 * PART || (o_stride % 8) != 0 || ((uintptr_t)out & 15) || window < 0 || !(scale > 0.f) ||
        n_seqs > 65535) return UB_ERR_ARG;
    LatentParams p;
    p.out = (bf16*)out; p.o_stride = o_stride; p.seq_start = seq_start; p.seq_before = seq_before; p.table = table;
    p.pages_per_seq = pages_per_seq; p.ring = ring; p.nh = nh; p.row = row; p.vals = vals; p.window = window;
    p.c = scale * LOG2E; p.sink = sink; p.error = error;
    p.part_o = part_o; p.part_ml = part_ml; p.n_slices = (!decode || n_slices < 1) ? 1 : n_slices;
    p.n_seqs = n_seqs; p.n_parts = (vals + PART - 1) / PART;
    const int tpb = BM / nh;
    p.n_row_tiles = (max_new + tpb - 1) / tpb;
    if (!decode) {
        const long long blocks = (long long)p.n_row_tiles * n_seqs * p.n_parts;
        if (blocks > 0x7fffffffll) return UB_ERR_ARG;
        return launch_latent<false>(dim3((unsigned)blocks), map_q, map_k, p, st);
    }
    if (max_new != 1) return UB_ERR_ARG;
    if (p.n_slices > 1 && (!part_o || !part_ml || ((uintptr_t)part_o & 15))) return UB_ERR_ARG;
    int rc = launch_latent<true>(dim3(p.n_slices, n_seqs, p.n_parts), map_q, map_k, p, st);
    if (rc != 0 || p.n_slices == 1) return rc;
    return (int)ub_launch_dependent(attn_latent_combine_kernel, dim3(n_seqs * nh), dim3(((vals / 4 + 31) / 32) * 32), 0, st, p);
}
