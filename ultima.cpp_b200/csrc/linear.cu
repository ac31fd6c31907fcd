// Recurrent layers whose state is, for every head, a matrix S [D, E] (D key channels, E value channels) in float32 that
// decays and takes up the token's key and value; nothing of what it holds enters the write:
//     S <- diag(a) S + k v^T;      o = S^T q
// Two forms of decay and gate:
//   channel  one decay a head and key channel, a = sigmoid(z)^(1 / tau), z = up(down(h)) + bias (gated linear attention)
//   head     exponential gates, one pair of numbers a head, with a running maximum m (the matrix memory): with the log
//            gates i = cap tanh(. / cap) and f = logsigmoid(cap tanh(. / cap)), m' = max(f + m, i), a = exp(f + m - m'),
//            the write times g = exp(i - m'); a vector n [D] is updated as S is with v = 1, and the read-out is divided by
//            max(|n.q|, exp(-m')) + 1e-6
// What the mixer puts out is o divided by its root mean square a head, times a weight (shared by the heads, or a row of all
// heads' size), times sigmoid or SiLU of an output gate's sums.
//
// The state of a sequence is a row of its slot: S [slots, H, D, E], n [slots, H, D], m [slots, H].  A step's tokens of one
// sequence are rows seq_start[s] .. seq_start[s + 1] of the packed batch.  Everything is float32; q, k, v and the gates come as
// columns of ONE projection row (float32 sums).
//
// Steps of several tokens a sequence:
//   lin_decay    (channel) the decays of every (token, head, channel), the low-rank product's second half included
//   lin_gates    (head) i, f, and the running maximum of a whole sequence by a scan of (max, +) over its tokens
//   lin_scan     the recurrence.  A long sequence is cut into chunks that are worked on side by side: a first pass leaves
//                every chunk's contribution to the state and its total decay, lin_carry turns them into the state before
//                every chunk, and a second pass makes the outputs.  (The state is linear in what came before, so this
//                costs the state's update twice and shortens the chain from token to token to a chunk's length.)
//   lin_finish   norm, weight, gate
// A step of one token a sequence is ONE kernel, lin_step: sums of the projection's K slices, gates, update, read-out, norm,
// weight, output gate.
#include "common.cuh"

__device__ __forceinline__ float sigmoid_(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float log_sigmoid_(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

struct LinShape {
    int H, D, E;             // heads, key size, value size
    int q_off, k_off, v_off, g_off;          // columns of a projection row
    int x_off, y_off;        // head form: the input and the forget gate's H columns; channel form: the low-rank columns, (unused)
    int rank;                // channel form: the number of low-rank columns
    int head_form;
    long long ldp;           // row stride of the projection
    int n_parts;             // the projection row is the sum of this many partial results ...
    long long part_stride;   // ... this many elements apart
};

__device__ __forceinline__ float lin_at(const float* __restrict__ p, const LinShape& s, long long t, int c) {
    float v = p[t * s.ldp + c];
    for (int i = 1; i < s.n_parts; ++i) v += p[i * s.part_stride + t * s.ldp + c];
    return v;
}

// ---------------------------------------------------------------------------------------
// decays a channel: dec[t, c] = exp(logsigmoid(sum_r low[t, r] up[r, c] + bias[c]) / tau); ``up`` [rank, H * D] float32
// ---------------------------------------------------------------------------------------
constexpr int DEC_TOK = 8;
constexpr int MAX_RANK = 512;

__global__ void __launch_bounds__(128)
lin_decay_kernel(const float* __restrict__ p, LinShape s, const float* __restrict__ up, const float* __restrict__ bias,
                 float* __restrict__ dec, int n_tokens, float inv_tau) {
    __shared__ float low[DEC_TOK][MAX_RANK];
    pdl_trigger();
    pdl_wait();
    const int t0 = blockIdx.x * DEC_TOK, n = min(DEC_TOK, n_tokens - t0);
    for (int i = threadIdx.x; i < DEC_TOK * s.rank; i += blockDim.x) {
        const int tt = i / s.rank, r = i % s.rank;
        low[tt][r] = tt < n ? lin_at(p, s, t0 + tt, s.x_off + r) : 0.f;
    }
    __syncthreads();
    const int C = s.H * s.D;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    float acc[DEC_TOK];
    const float b = bias[c];
#pragma unroll
    for (int tt = 0; tt < DEC_TOK; ++tt) acc[tt] = 0.f;
    for (int r = 0; r < s.rank; ++r) {
        const float w = up[(long long)r * C + c];
#pragma unroll
        for (int tt = 0; tt < DEC_TOK; ++tt) acc[tt] = fmaf(w, low[tt][r], acc[tt]);
    }
#pragma unroll
    for (int tt = 0; tt < DEC_TOK; ++tt)
        if (tt < n) dec[(long long)(t0 + tt) * C + c] = expf(log_sigmoid_(acc[tt] + b) * inv_tau);
}

// ---------------------------------------------------------------------------------------
// exponential gates: keep = exp(f + m_before - m), put = exp(i - m), floor = exp(-m), [T, H] each; one block a (sequence, head)
// ---------------------------------------------------------------------------------------
constexpr int GATE_WARPS = 16;

__device__ __forceinline__ void log_gates(float zi, float zf, float cap, float& i, float& f) {
    i = cap * tanhf(zi / cap);
    f = log_sigmoid_(cap * tanhf(zf / cap));
}

__global__ void __launch_bounds__(GATE_WARPS * 32)
lin_gates_kernel(const float* __restrict__ p, LinShape s, const float* __restrict__ bi, const float* __restrict__ bf, float cap,
                 float* __restrict__ m_state, const int* __restrict__ seq_start, const int* __restrict__ seq_slot,
                 float* __restrict__ keep, float* __restrict__ put, float* __restrict__ floor_) {
    // A token maps the maximum before it, m, to max(f + m, i): two such maps in a row are (f1 + f2, max(f2 + i1, i2)).
    __shared__ float wf[GATE_WARPS], wi[GATE_WARPS];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t0 = seq_start[b], t1 = seq_start[b + 1];
    if (t0 >= t1) return;
    float* ms = m_state + (long long)seq_slot[b] * s.H + h;
    float m = *ms;                                            // the maximum before this turn's first token
    const float b_in = bi[h], b_forget = bf[h];
    float zi = 0.f, zf = 0.f;                                 // a turn's sums are asked for while the turn before it is worked on
    auto ask = [&](int t) {
        if (t < t1) { zi = lin_at(p, s, t, s.x_off + h); zf = lin_at(p, s, t, s.y_off + h); }
    };
    ask(t0 + threadIdx.x);
    for (int base = t0; base < t1; base += GATE_WARPS * 32) {
        const int t = base + threadIdx.x;
        const float yi = zi, yf = zf;
        ask(t + GATE_WARPS * 32);
        float f1 = 0.f, i1 = -INFINITY;                       // past the end: the map that changes nothing
        if (t < t1) log_gates(yi + b_in, yf + b_forget, cap, i1, f1);
        float f = f1, i = i1;                                 // the map of this warp's tokens up to and with this lane's
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pf = __shfl_up_sync(0xffffffffu, f, o), pi = __shfl_up_sync(0xffffffffu, i, o);
            if (lane >= o) { i = fmaxf(f + pi, i); f += pf; }
        }
        if (lane == 31) { wf[warp] = f; wi[warp] = i; }
        __syncthreads();
        float mb = m;                                         // the maximum before this warp's first token
        for (int w = 0; w < warp; ++w) mb = fmaxf(wf[w] + mb, wi[w]);
        const float now = fmaxf(f + mb, i);
        float before = __shfl_up_sync(0xffffffffu, now, 1);
        if (lane == 0) before = mb;
        if (t < t1) {
            const long long o = (long long)t * s.H + h;
            keep[o] = expf(f1 + before - now);
            put[o] = expf(i1 - now);
            floor_[o] = expf(-now);
        }
        for (int w = 0; w < GATE_WARPS; ++w) m = fmaxf(wf[w] + m, wi[w]);      // (the same for every thread)
        __syncthreads();
    }
    if (threadIdx.x == 0) *ms = m;
}

// ---------------------------------------------------------------------------------------
// the recurrence over a chunk of a sequence
// ---------------------------------------------------------------------------------------
__device__ __forceinline__ void lin_cp4(float* dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void lin_cp16(float* dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
// Two float32 in a 64-bit register and the arithmetic on such pairs (one instruction for both).
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
__device__ __forceinline__ uint64_t mul_pair(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// LANES lanes share a column of S, each with R of its D channels; a thread holds C neighbouring columns, which share its reads
// of the token's q, k and decays (those reads and the arithmetic are about equally dear).
template <int LANES, int R, int C, bool HEAD>
struct ScanLayout {
    static constexpr int DP = LANES * R, COLS = 128 / LANES * C;
    static constexpr int TT = DP <= 128 ? 8 : 4;              // tokens a stage
    static constexpr int STAGES = 3;
    static constexpr int BLOCKS = R <= 4 ? 4 : 3;             // blocks an SM the registers are cut for
    static constexpr int TOKEN = (HEAD ? 2 : 3) * DP + COLS + 4;      // floats of a token: q, k, (decays), v, (keep, put)
    static constexpr size_t BYTES = (size_t)STAGES * TT * TOKEN * sizeof(float);
};

// The sum over a column's LANES lanes of C values each: every exchange halves the values a lane is left with, so a lane ends
// with the sum of value ``sum_of``.
template <int LANES, int C>
__device__ __forceinline__ float lane_sums(float (&o)[C], int l) {
    int mask = LANES / 2;
#pragma unroll
    for (int n = C / 2; n >= 1; n >>= 1, mask >>= 1) {
        const bool up = l & mask;
#pragma unroll
        for (int x = 0; x < n; ++x) {
            const float mine = up ? o[x + n] : o[x], other = up ? o[x] : o[x + n];
            o[x] = mine + __shfl_xor_sync(0xffffffffu, other, mask);
        }
    }
    float r = o[0];
#pragma unroll
    for (; mask >= 1; mask >>= 1) r += __shfl_xor_sync(0xffffffffu, r, mask);
    return r;
}

struct ScanParams {
    const float* p;
    const float* dec;                         // channel form: decays [T, H * D]; head form: keep [T, H]
    const float* put;                         // head form: [T, H]
    float* out; int EW;                       // [T, H, EW]; EW = E, or E + 1 with n.q in the last column (head form)
    float* S; float* n;                       // the slots' state
    float* work;                              // [chunks][seqs][H][D][EW]: chunk contributions, then the states before the chunks
    float* decay;                             // [chunks][seqs][H][D] (head form: [..][H]): a chunk's total decay
    const int* seq_start; const int* seq_slot;
    int n_seqs, n_chunks, chunk;
};

enum { SCAN_WHOLE = 0, SCAN_SUM = 1, SCAN_OUT = 2 };

// Grid (blocks of columns, heads, sequences * chunks), 128 threads.  SCAN_WHOLE: one chunk, from the slot's state to the slot's
// state.  SCAN_SUM: from zero, no output; leaves the chunk's contribution and its total decay.  SCAN_OUT: from the state
// before the chunk (work); the last chunk leaves the slot's state.
// A thread holds C neighbouring columns of S and of each the channels of the float4 chunks l, l + LANES, ... (l its lane among the
// column's): the lanes read consecutive bytes of shared memory, and all columns of a warp the same ones.  Tokens come
// through shared memory a stage at a time, the next stages on their way while one is worked on.
template <int LANES, int R, int C, bool HEAD, bool VEC, int PASS>
__global__ void __launch_bounds__(128, (ScanLayout<LANES, R, C, HEAD>::BLOCKS))
lin_scan_kernel(ScanParams a, LinShape s) {
    using L = ScanLayout<LANES, R, C, HEAD>;
    constexpr int DP = L::DP, COLS = L::COLS, TT = L::TT, NC = R / 4, ST = L::STAGES;
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;                                            // [ST][TT][DP]
    float* sk = sq + ST * TT * DP;
    float* sa = sk + ST * TT * DP;                             // (channel form)
    float* sv = sa + (HEAD ? 0 : ST * TT * DP);                // [ST][TT][COLS]
    float* sg = sv + ST * TT * COLS;                           // [ST][TT][4]: keep, put (head form)
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, l = tid % LANES, warp = tid >> 5;
    const int col = tid / LANES * C;                      // the first of this thread's columns in the block
    const int h = blockIdx.y, b = blockIdx.z % a.n_seqs, ck = blockIdx.z / a.n_seqs;
    const int D = s.D, E = s.E, EW = a.EW, H = s.H;
    const int j0 = blockIdx.x * COLS, j = j0 + col;
    const int s0 = a.seq_start[b], s1 = a.seq_start[b + 1];
    const int t0 = PASS == SCAN_WHOLE ? s0 : s0 + ck * a.chunk;
    const int t1 = PASS == SCAN_WHOLE ? s1 : min(s1, t0 + a.chunk);
    if (t0 >= t1) return;                                      // (the whole block)
    if (PASS == SCAN_SUM && t1 == s1) return;                  // nothing follows the last chunk
    const long long slot = a.seq_slot[b];
    float* Sh = a.S + (slot * H + h) * D * E;
    float* nh = a.n ? a.n + (slot * H + h) * D : nullptr;
    float* Wh = PASS == SCAN_WHOLE ? nullptr : a.work + (((long long)ck * a.n_seqs + b) * H + h) * D * EW;

    uint64_t st[NC][2][C];                                     // pairs of neighbouring channels of a column
    auto place = [&](int d, int jj) -> float* {                // where S (and n) of the slot has (channel, column)
        return jj < E ? Sh + (long long)d * E + jj : nh + d;
    };
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int d = (c * LANES + l) * 4 + 2 * u;
#pragma unroll
            for (int x = 0; x < C; ++x) {
                float v0 = 0.f, v1 = 0.f;
                if (PASS != SCAN_SUM && j + x < EW) {
                    if (d < D) v0 = PASS == SCAN_WHOLE ? *place(d, j + x) : Wh[(long long)d * EW + j + x];
                    if (d + 1 < D) v1 = PASS == SCAN_WHOLE ? *place(d + 1, j + x) : Wh[(long long)(d + 1) * EW + j + x];
                }
                st[c][u][x] = pair_of(v0, v1);
            }
        }
    // channels and columns past the sizes are constants that no copy ever touches; the column behind the values is 1
    for (int i = tid; i < ST * TT * DP; i += blockDim.x)
        if (i % DP >= D) { sq[i] = 0.f; sk[i] = 0.f; if (!HEAD) sa[i] = 1.f; }
    for (int i = tid; i < ST * TT * COLS; i += blockDim.x) {
        const int jj = j0 + i % COLS;
        if (jj >= E) sv[i] = (jj == E && EW > E) ? 1.f : 0.f;
    }
    const float* prow = a.p + (long long)h * D;
    // one group of copies is committed for every stage, empty past the end, so the count to wait for is fixed
    auto fetch = [&](int base, int buf) {
        const int cnt = max(0, min(TT, t1 - base));
        const int vcols = min(COLS, E - j0);                   // (<= 0: this block has the column behind the values only)
        if (VEC) {
            const int n4 = D >> 2;
            for (int i = tid; i < cnt * n4; i += blockDim.x) {
                const int tt = i / n4, d = (i % n4) * 4;
                const long long row = (long long)(base + tt) * s.ldp;
                if (PASS != SCAN_SUM) lin_cp16(sq + (buf * TT + tt) * DP + d, prow + row + s.q_off + d);
                lin_cp16(sk + (buf * TT + tt) * DP + d, prow + row + s.k_off + d);
                if (!HEAD) lin_cp16(sa + (buf * TT + tt) * DP + d, a.dec + ((long long)(base + tt) * H + h) * D + d);
            }
            const int v4 = vcols > 0 ? vcols >> 2 : 0;
            for (int i = tid; i < cnt * v4; i += blockDim.x) {
                const int tt = i / v4, c = (i % v4) * 4;
                lin_cp16(sv + (buf * TT + tt) * COLS + c, a.p + (long long)(base + tt) * s.ldp + s.v_off + (long long)h * E + j0 + c);
            }
        } else {
            for (int i = tid; i < cnt * D; i += blockDim.x) {
                const int tt = i / D, d = i % D;
                const long long row = (long long)(base + tt) * s.ldp;
                if (PASS != SCAN_SUM) lin_cp4(sq + (buf * TT + tt) * DP + d, prow + row + s.q_off + d);
                lin_cp4(sk + (buf * TT + tt) * DP + d, prow + row + s.k_off + d);
                if (!HEAD) lin_cp4(sa + (buf * TT + tt) * DP + d, a.dec + ((long long)(base + tt) * H + h) * D + d);
            }
            for (int i = tid; i < cnt * max(vcols, 0); i += blockDim.x) {
                const int tt = i / vcols, c = i % vcols;
                lin_cp4(sv + (buf * TT + tt) * COLS + c, a.p + (long long)(base + tt) * s.ldp + s.v_off + (long long)h * E + j0 + c);
            }
        }
        if (HEAD && tid < cnt) {
            lin_cp4(sg + (buf * TT + tid) * 4, a.dec + (long long)(base + tid) * H + h);
            lin_cp4(sg + (buf * TT + tid) * 4 + 1, a.put + (long long)(base + tid) * H + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const bool busy = j0 + warp * (32 / LANES) * C < EW;  // a warp whose columns lie past the end only helps fetching
    const bool sums_decay = PASS == SCAN_SUM && blockIdx.x == 0;       // the chunk's total decay: of channels tid and tid + 128, or of the head
    float total[2] = {1.f, 1.f};
    // behind the exchange a lane holds the sum of one of the C columns: the bits of its number from the top
    constexpr int SPARE = LANES / C;                           // lanes that end with the same column
    int my_x = 0;
#pragma unroll
    for (int n = C / 2, mask = LANES / 2; n >= 1; n >>= 1, mask >>= 1) my_x += (l & mask) ? n : 0;
    const bool stores = l % SPARE == 0;

#pragma unroll
    for (int i = 0; i < ST - 1; ++i) fetch(t0 + i * TT, i);
    int buf = 0;
    for (int base = t0; base < t1; base += TT, buf = buf + 1 == ST ? 0 : buf + 1) {
        const int cnt = min(TT, t1 - base);
        asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
        __syncthreads();                                       // this stage is there, and nobody reads the one before it any more
        fetch(base + (ST - 1) * TT, buf == 0 ? ST - 1 : buf - 1);
        auto token = [&](int tt) {
            const float* vt = sv + (buf * TT + tt) * COLS + col;
            float v[C];
#pragma unroll
            for (int x = 0; x < C; ++x) v[x] = vt[x];
            uint64_t keep2 = 0;
            if (HEAD) {
                const float2 g = *reinterpret_cast<const float2*>(sg + (buf * TT + tt) * 4);
                keep2 = pair_of(g.x, g.x);
#pragma unroll
                for (int x = 0; x < C; ++x) v[x] *= g.y;
            }
            uint64_t v2[C], o2[C];
#pragma unroll
            for (int x = 0; x < C; ++x) { v2[x] = pair_of(v[x], v[x]); o2[x] = 0; }
            const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(sq + (buf * TT + tt) * DP);
            const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(sk + (buf * TT + tt) * DP);
            const ulonglong2* a4 = reinterpret_cast<const ulonglong2*>(sa + (buf * TT + tt) * DP);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const ulonglong2 kk = k4[c * LANES + l];
                ulonglong2 qq, aa;
                if (PASS != SCAN_SUM) qq = q4[c * LANES + l];
                if (!HEAD) aa = a4[c * LANES + l];
                const uint64_t k2[2] = {kk.x, kk.y};
                const uint64_t a2[2] = {HEAD ? keep2 : aa.x, HEAD ? keep2 : aa.y};
#pragma unroll
                for (int u = 0; u < 2; ++u) {
#pragma unroll
                    for (int x = 0; x < C; ++x) {
                        st[c][u][x] = fma_pair(a2[u], st[c][u][x], mul_pair(k2[u], v2[x]));
                        if (PASS != SCAN_SUM) o2[x] = fma_pair(st[c][u][x], u ? qq.y : qq.x, o2[x]);
                    }
                }
            }
            if (PASS != SCAN_SUM) {
                float o[C];
#pragma unroll
                for (int x = 0; x < C; ++x) { float lo, hi; halves_of(o2[x], lo, hi); o[x] = lo + hi; }
                const float r = lane_sums<LANES, C>(o, l);
                if (stores && j + my_x < EW) a.out[((long long)(base + tt) * H + h) * EW + j + my_x] = r;
            }
        };
        if (PASS == SCAN_SUM && sums_decay) {
            for (int tt = 0; tt < cnt; ++tt) {
                if (HEAD) total[0] *= sg[(buf * TT + tt) * 4];
                else {
                    if (tid < DP) total[0] *= sa[(buf * TT + tt) * DP + tid];
                    if (DP > 128 && tid + 128 < DP) total[1] *= sa[(buf * TT + tt) * DP + tid + 128];
                }
            }
        }
        if (busy) {
            if (cnt == TT) {
#pragma unroll
                for (int tt = 0; tt < TT; ++tt) token(tt);
            } else {
                for (int tt = 0; tt < cnt; ++tt) token(tt);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (PASS == SCAN_SUM && sums_decay) {
        float* P = a.decay + (((long long)ck * a.n_seqs + b) * H + h) * (HEAD ? 1 : D);
        if (HEAD) { if (tid == 0) *P = total[0]; }
        else {
            if (tid < D) P[tid] = total[0];
            if (tid + 128 < D) P[tid + 128] = total[1];
        }
    }
    if (!busy || (PASS == SCAN_OUT && t1 != s1)) return;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int d = (c * LANES + l) * 4 + 2 * u;
#pragma unroll
            for (int x = 0; x < C; ++x) {
                float v0, v1;
                halves_of(st[c][u][x], v0, v1);
                if (j + x >= EW) continue;
                if (d < D) *(PASS == SCAN_SUM ? Wh + (long long)d * EW + j + x : place(d, j + x)) = v0;
                if (d + 1 < D) *(PASS == SCAN_SUM ? Wh + (long long)(d + 1) * EW + j + x : place(d + 1, j + x)) = v1;
            }
        }
}

// Chunk contributions -> the state before every chunk, in place: one thread a (sequence, head, channel, column).
__global__ void __launch_bounds__(256)
lin_carry_kernel(ScanParams a, int H, int D, int E, int head_form) {
    pdl_trigger();
    pdl_wait();
    const long long per_seq = (long long)H * D * a.EW;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= per_seq * a.n_seqs) return;
    const int b = (int)(i / per_seq);
    const long long r = i % per_seq;
    const int jj = (int)(r % a.EW);
    const long long hd = r / a.EW;                             // head * D + channel
    const int len = a.seq_start[b + 1] - a.seq_start[b];
    const int n = (len + a.chunk - 1) / a.chunk;
    if (n == 0) return;
    const long long slot = a.seq_slot[b];
    float s = jj < E ? a.S[(slot * H * D + hd) * E + jj] : a.n[slot * H * D + hd];
    const long long step = per_seq * a.n_seqs;
    float* w = a.work + i;
    const long long dstep = (long long)a.n_seqs * H * (head_form ? 1 : D);
    const float* dc = a.decay + (long long)b * H * (head_form ? 1 : D) + (head_form ? hd / D : hd);
    int c = 0;
    for (; c + 4 < n; c += 4) {                                // (chunk n - 1 has left nothing)
        float add[4], dec[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) { add[u] = w[(c + u) * step]; dec[u] = dc[(c + u) * dstep]; }
#pragma unroll
        for (int u = 0; u < 4; ++u) { w[(c + u) * step] = s; s = fmaf(dec[u], s, add[u]); }
    }
    for (; c < n; ++c) {
        if (c == n - 1) { w[c * step] = s; break; }
        const float add = w[c * step], dec = dc[c * dstep];
        w[c * step] = s;
        s = fmaf(dec, s, add);
    }
}

// ---------------------------------------------------------------------------------------
// what leaves the mixer: one warp a (token, head)
// ---------------------------------------------------------------------------------------
template <typename TO>
__global__ void __launch_bounds__(128)
lin_finish_kernel(const float* __restrict__ o, int EW, const float* __restrict__ p, LinShape s, const float* __restrict__ floor_,
                  const float* __restrict__ w, int w_heads, int silu_gate, TO* __restrict__ out, int n_tokens, float q_scale,
                  float eps, float out_scale) {
    pdl_trigger();
    pdl_wait();
    const long long wid = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (wid >= (long long)n_tokens * s.H) return;
    const long long t = wid / s.H;
    const int h = (int)(wid % s.H), E = s.E;
    const float* orow = o + wid * EW;
    float factor = q_scale;
    if (s.head_form) factor = q_scale / (fmaxf(fabsf(q_scale * orow[E]), floor_[wid]) + 1e-6f);
    constexpr int KEEP = 8;                                    // values a lane keeps between the passes
    float v[KEEP], zk[KEEP];
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {                           // (the gate's sums are asked for together with the values)
        const int e = lane + 32 * u;
        v[u] = e < E ? orow[e] : 0.f;
        zk[u] = e < E ? p[t * s.ldp + s.g_off + h * E + e] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {
        v[u] *= factor;
        ss = fmaf(v[u], v[u], ss);
    }
    for (int e = lane + 32 * KEEP; e < E; e += 32) { const float x = orow[e] * factor; ss = fmaf(x, x, ss); }
    const float inv = inv_rms(warp_sum(ss), (float)E, eps) * out_scale;
    if (w_heads) w += (long long)h * E;
    auto put = [&](int e, float x, float z) {
        const float g = sigmoid_(z);
        out[wid * E + e] = from_f32<TO>(x * inv * w[e] * (silu_gate ? z * g : g));
    };
#pragma unroll
    for (int u = 0; u < KEEP; ++u) {
        const int e = lane + 32 * u;
        if (e < E) put(e, v[u], zk[u]);
    }
    for (int e = lane + 32 * KEEP; e < E; e += 32) put(e, orow[e] * factor, p[t * s.ldp + s.g_off + h * E + e]);
}

// ---------------------------------------------------------------------------------------
// one token a sequence: everything between the input product and the output product in one kernel
// ---------------------------------------------------------------------------------------
struct StepParams {
    const float* p;
    const float* up; const float* bias; float inv_tau;                     // channel form
    const float* bi; const float* bf; float cap;                           // head form
    float* S; float* n; float* m;
    const int* seq_start; const int* seq_slot;
    const float* w; int w_heads, silu_gate;
    void* out;
    float q_scale, eps, out_scale;
};

constexpr int STEP_THREADS = 256;
constexpr int STEP_AHEAD = 8;                 // 16-byte pieces of the state a thread asks for before the kernel ahead has ended
constexpr int STEP_PARTS = 8;                 // the most blocks that share a head (a cluster)

__device__ __forceinline__ void cluster_meet() {
    asm volatile("barrier.cluster.arrive.release;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire;" ::: "memory");
}
// the float at ``p`` (shared memory) of the cluster's block ``rank``
__device__ __forceinline__ float cluster_read(const float* p, int rank) {
    uint32_t a;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"((uint32_t)__cvta_generic_to_shared(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
    return v;
}

// Grid (parts, heads, sequences), clusters of ``parts`` blocks: a block takes ``cols`` columns of its head's S.  The blocks of a
// cluster meet once, for the sum of squares over the whole head; what they all need (q, k, gates, n.q) each works out itself, and
// the first one writes n and m once the others have read them.
template <typename TO, bool VEC>
__global__ void __launch_bounds__(STEP_THREADS, 2)
lin_step_kernel(StepParams a, LinShape s, int cols) {
    constexpr int W = VEC ? 4 : 1;
    extern __shared__ __align__(16) float sm[];
    const int D = s.D, H = s.H, parts = gridDim.x, part = blockIdx.x;
    const int c0 = part * cols, E = min(cols, s.E - c0);       // this block's columns
    const int EP = (cols + 3) / 4 * 4, ER = (E + 3) / 4 * 4;
    float* sq = sm;                            // [D]
    float* sk = sq + D;                        // [D]
    float* sa = sk + D;                        // [D] decays (channel form)
    float* sv = sa + D + (4 - 3 * D % 4) % 4;  // [EP]
    float* sz = sv + EP;                       // [EP] the output gate's sums
    float* red = sz + EP;                      // [groups][ER]: at most max(4 * STEP_THREADS, EP) numbers
    __shared__ float rs[40], low[MAX_RANK], shared_ss;
    pdl_trigger();
    const int tid = threadIdx.x, h = blockIdx.y, b = blockIdx.z;
    const long long slot = a.seq_slot[b];
    const long long t = a.seq_start[b];
    float* Sh = a.S + (slot * H + h) * D * s.E + c0;
    float* nh = s.head_form ? a.n + (slot * H + h) * D : nullptr;
    const int ne = E / W;                      // pieces of a row of this block's columns
    const int per = max(1, min(ne, STEP_THREADS));             // threads on one row
    const int groups = STEP_THREADS / per;     // rows side by side
    const int grp = tid / per, e0 = tid % per;
    const bool works = grp < groups && ne > 0;
    // the state was left by an earlier step: its first pieces are asked for while the kernel ahead still runs
    alignas(16) float ahead[STEP_AHEAD][W];
    if (works) {
#pragma unroll
        for (int u = 0; u < STEP_AHEAD; ++u) {
            const int d = grp + u * groups;
            if (d < D) {
                if (VEC) *reinterpret_cast<float4*>(ahead[u]) = *reinterpret_cast<const float4*>(Sh + (long long)d * s.E + e0 * W);
                else ahead[u][0] = Sh[(long long)d * s.E + e0];
            }
        }
    }
    const float n_old = (s.head_form && tid < D) ? nh[tid] : 0.f;              // (D <= 256: a channel a thread)
    const float m_old = s.head_form ? a.m[slot * H + h] : 0.f;
    static_assert(STEP_THREADS >= 256, "a key channel a thread");
    pdl_wait();
    // everything this block needs of the projection row, several numbers a thread asked for before the first is put away:
    // q, k, this block's columns of v and of the output gate, and the gates' sums or the low-rank columns
    const int n_low = s.head_form ? 2 : s.rank, total = 2 * D + 2 * E + n_low;
    auto column = [&](int i, float*& dst) -> int {
        if (i < D) { dst = sq + i; return s.q_off + h * D + i; }
        i -= D;
        if (i < D) { dst = sk + i; return s.k_off + h * D + i; }
        i -= D;
        if (i < E) { dst = sv + i; return s.v_off + h * s.E + c0 + i; }
        i -= E;
        if (i < E) { dst = sz + i; return s.g_off + h * s.E + c0 + i; }
        i -= E;
        dst = low + i;
        return s.head_form ? (i == 0 ? s.x_off : s.y_off) + h : s.x_off + i;
    };
    for (int i0 = tid; i0 < total; i0 += 4 * STEP_THREADS) {
        float v[4];
        float* dst[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int i = i0 + u * STEP_THREADS;
            dst[u] = nullptr;
            if (i < total) v[u] = lin_at(a.p, s, t, column(i, dst[u]));
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (dst[u]) *dst[u] = v[u];
    }
    __syncthreads();
    float keep = 1.f, put = 1.f, floor_ = 0.f;
    if (s.head_form) {
        if (tid == 0) {
            float li, lf;
            log_gates(low[0] + a.bi[h], low[1] + a.bf[h], a.cap, li, lf);
            const float m_new = fmaxf(lf + m_old, li);
            rs[34] = expf(lf + m_old - m_new);
            rs[35] = expf(li - m_new);
            rs[36] = expf(-m_new);
            rs[37] = m_new;
        }
    }
    if (!s.head_form) {
        for (int d = tid; d < D; d += STEP_THREADS) {
            const int c = h * D + d;
            float z = 0.f;
#pragma unroll 8
            for (int r = 0; r < s.rank; ++r) z = fmaf(a.up[(long long)r * H * D + c], low[r], z);
            sa[d] = expf(log_sigmoid_(z + a.bias[c]) * a.inv_tau);
        }
    }
    __syncthreads();
    if (s.head_form) { keep = rs[34]; put = rs[35]; floor_ = rs[36]; }
    // the vector n and its product with q
    float nq = 0.f, n_new = 0.f;
    if (s.head_form) {
        if (tid < D) {
            n_new = fmaf(keep, n_old, put * sk[tid]);
            nq = n_new * sq[tid];
        }
        nq = block_sum(nq, rs);
    }
    // S, a row at a time in every group; rows wider than the block in several turns
    for (int eb = 0; eb < ne; eb += per) {
        const int ee = eb + e0;
        if (works && ee < ne) {
            float acc[W], v[W];
#pragma unroll
            for (int x = 0; x < W; ++x) { acc[x] = 0.f; v[x] = sv[ee * W + x] * put; }
            auto row = [&](int d, float* x) {
                const float k = sk[d], q = sq[d], dk = s.head_form ? keep : sa[d];
#pragma unroll
                for (int y = 0; y < W; ++y) {
                    x[y] = fmaf(dk, x[y], k * v[y]);
                    acc[y] = fmaf(x[y], q, acc[y]);
                }
                if (VEC) *reinterpret_cast<float4*>(Sh + (long long)d * s.E + ee * W) = *reinterpret_cast<float4*>(x);
                else Sh[(long long)d * s.E + ee] = x[0];
            };
            int d = grp;
            if (eb == 0) {
#pragma unroll
                for (int u = 0; u < STEP_AHEAD; ++u) {
                    if (d < D) row(d, ahead[u]);
                    d += groups;
                }
            }
            for (; d < D; d += 8 * groups) {
                alignas(16) float x[8][W];
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const int dd = d + u * groups;
                    if (dd < D) {
                        if (VEC) *reinterpret_cast<float4*>(x[u]) = *reinterpret_cast<const float4*>(Sh + (long long)dd * s.E + ee * W);
                        else x[u][0] = Sh[(long long)dd * s.E + ee];
                    }
                }
#pragma unroll
                for (int u = 0; u < 8; ++u)
                    if (d + u * groups < D) row(d + u * groups, x[u]);
            }
#pragma unroll
            for (int y = 0; y < W; ++y) red[grp * ER + ee * W + y] = acc[y];
        }
    }
    __syncthreads();
    float factor = a.q_scale;
    if (s.head_form) factor = a.q_scale / (fmaxf(fabsf(a.q_scale * nq), floor_) + 1e-6f);
    float ss = 0.f;
    for (int e = tid; e < E; e += STEP_THREADS) {
        float o = 0.f;
        for (int g = 0; g < groups; ++g) o += red[g * ER + e];
        o *= factor;
        sv[e] = o;                              // (v is used up)
        ss = fmaf(o, o, ss);
    }
    ss = block_sum(ss, rs);
    if (parts > 1) {
        if (tid == 0) shared_ss = ss;
        cluster_meet();                         // every block's share is there, and every block has read n and m
        ss = 0.f;
        for (int r = 0; r < parts; ++r) ss += cluster_read(&shared_ss, r);
    }
    if (s.head_form && part == 0) {
        if (tid < D) nh[tid] = n_new;
        if (tid == 0) a.m[slot * H + h] = rs[37];
    }
    const float inv = inv_rms(ss, (float)s.E, a.eps) * a.out_scale;
    const float* w = a.w + (a.w_heads ? (long long)h * s.E : 0) + c0;
    TO* out = (TO*)a.out + (t * H + h) * s.E + c0;
    for (int e = tid; e < E; e += STEP_THREADS) {
        const float z = sz[e], g = sigmoid_(z);
        out[e] = from_f32<TO>(sv[e] * inv * w[e] * (a.silu_gate ? z * g : g));
    }
    if (parts > 1) cluster_meet();              // no block leaves while another may still read its share
}

// ---------------------------------------------------------------------------------------
// shape: [H, D, E, q_off, k_off, v_off, g_off, x_off, y_off, rank, head_form] (11 ints)
static int read_shape(const int* q, long long ldp, int n_parts, long long part_stride, LinShape& s) {
    s.H = q[0]; s.D = q[1]; s.E = q[2]; s.q_off = q[3]; s.k_off = q[4]; s.v_off = q[5]; s.g_off = q[6]; s.x_off = q[7];
    s.y_off = q[8]; s.rank = q[9]; s.head_form = q[10];
    s.ldp = ldp; s.n_parts = n_parts; s.part_stride = part_stride;
    if (s.H <= 0 || s.D <= 0 || s.D > 256 || s.E <= 0 || s.E > 1024 || s.H > 65535 || n_parts < 1) return UB_ERR_ARG;
    if (!s.head_form && (s.rank < 1 || s.rank > MAX_RANK)) return UB_ERR_ARG;
    if (s.q_off < 0 || s.k_off < 0 || s.v_off < 0 || s.g_off < 0 || s.x_off < 0) return UB_ERR_ARG;
    return 0;
}

UB_API int ub_lin_decay(const float* p, long long ldp, int n_parts, long long part_stride, const int* shape, const float* up,
                        const float* bias, float* dec, int n_tokens, float tau, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    LinShape s;
    if (int rc = read_shape(shape, ldp, n_parts, part_stride, s)) return rc;
    if (s.head_form || !(tau > 0.f)) return UB_ERR_ARG;
    const dim3 grid((n_tokens + DEC_TOK - 1) / DEC_TOK, (s.H * s.D + 127) / 128);
    return (int)ub_launch_dependent(lin_decay_kernel, grid, dim3(128), 0, st, p, s, up, bias, dec, n_tokens, 1.0f / tau);
}

UB_API int ub_lin_gates(const float* p, long long ldp, int n_parts, long long part_stride, const int* shape, const float* bi,
                        const float* bf, float cap, float* m, const int* seq_start, const int* seq_slot, int n_seqs, float* keep,
                        float* put, float* floor_, cudaStream_t st) {
    if (n_seqs <= 0) return 0;
    LinShape s;
    if (int rc = read_shape(shape, ldp, n_parts, part_stride, s)) return rc;
    if (!s.head_form || !(cap > 0.f) || n_seqs > 65535) return UB_ERR_ARG;
    return (int)ub_launch_dependent(lin_gates_kernel, dim3(s.H, n_seqs), dim3(GATE_WARPS * 32), 0, st, p, s, bi, bf, cap, m,
                                    seq_start, seq_slot, keep, put, floor_);
}

template <int LANES, int R, int C, bool HEAD, bool VEC, int PASS>
static cudaError_t launch_scan(const ScanParams& a, const LinShape& s, cudaStream_t st) {
    using L = ScanLayout<LANES, R, C, HEAD>;
    static bool attr_done = false;
    if (!attr_done && L::BYTES > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(lin_scan_kernel<LANES, R, C, HEAD, VEC, PASS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)L::BYTES);
        if (e != cudaSuccess) return e;
        attr_done = true;
    }
    const int chunks = PASS == SCAN_WHOLE ? 1 : a.n_chunks;
    const dim3 grid((a.EW + L::COLS - 1) / L::COLS, s.H, a.n_seqs * chunks);
    // an ordinary launch: as a programmatic dependent the blocks, each busy for the whole kernel, would be placed several to an
    // SM on the SMs that the kernel before leaves first
    return ub_launch_ordered(false, lin_scan_kernel<LANES, R, C, HEAD, VEC, PASS>, grid, dim3(128), L::BYTES, st, a, s);
}

template <int LANES, int R, int C, bool HEAD, bool VEC>
static cudaError_t scan_all(const ScanParams& a, const LinShape& s, cudaStream_t st) {
    if (a.n_chunks <= 1) return launch_scan<LANES, R, C, HEAD, VEC, SCAN_WHOLE>(a, s, st);
    cudaError_t e = launch_scan<LANES, R, C, HEAD, VEC, SCAN_SUM>(a, s, st);
    if (e != cudaSuccess) return e;
    const long long n = (long long)a.n_seqs * s.H * s.D * a.EW;
    e = ub_launch_dependent(lin_carry_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, a, s.H, s.D, s.E, s.head_form);
    if (e != cudaSuccess) return e;
    return launch_scan<LANES, R, C, HEAD, VEC, SCAN_OUT>(a, s, st);
}

// The projection whole (one part).  ``n_chunks`` chunks of ``chunk`` tokens cover the longest sequence (1: no chunks; work and
// decay are then not used).
UB_API int ub_lin_scan(const float* p, long long ldp, const int* shape, const float* dec, const float* put, float* out, float* S,
                       float* n, float* work, float* decay, const int* seq_start, const int* seq_slot, int n_seqs, int n_chunks,
                       int chunk, cudaStream_t st) {
    if (n_seqs <= 0) return 0;
    LinShape s;
    if (int rc = read_shape(shape, ldp, 1, 0, s)) return rc;
    if (s.head_form ? (!put || !n) : (put != nullptr)) return UB_ERR_ARG;
    if (n_chunks > 1 && (!work || !decay || chunk < 1)) return UB_ERR_ARG;
    if (n_chunks < 1 || (long long)n_seqs * n_chunks > 65535) return UB_ERR_ARG;
    ScanParams a{p, dec, put, out, s.head_form ? s.E + 1 : s.E, S, s.head_form ? n : nullptr, work, decay, seq_start, seq_slot,
                 n_seqs, n_chunks, chunk};
    const bool vec = s.D % 4 == 0 && s.E % 4 == 0 && ldp % 4 == 0 && (s.q_off | s.k_off | s.v_off) % 4 == 0 &&
        (((uintptr_t)p | (uintptr_t)(s.head_form ? nullptr : dec)) & 15) == 0;
    cudaError_t e;
#define GO2(LL, RR, CC, HH) e = vec ? scan_all<LL, RR, CC, HH, true>(a, s, st) : scan_all<LL, RR, CC, HH, false>(a, s, st)
#define GO(LL, RR, CC) do { if (s.head_form) GO2(LL, RR, CC, true); else GO2(LL, RR, CC, false); } while (0)
    if (s.D <= 32) GO(8, 4, 8);                                // (blocks of 128 columns, 128, 64 and 32: lin_chunks counts them)
    else if (s.D <= 64) GO(8, 8, 8);
    else if (s.D <= 128) GO(8, 16, 4);
    else GO(32, 8, 8);
#undef GO
#undef GO2
    return (int)e;
}

UB_API int ub_lin_finish(const float* o, const float* p, long long ldp, const int* shape, const float* floor_, const float* w,
                         int w_heads, int silu_gate, void* out, int out_dtype, int n_tokens, float q_scale, float eps,
                         float out_scale, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    LinShape s;
    if (int rc = read_shape(shape, ldp, 1, 0, s)) return rc;
    if (s.head_form && !floor_) return UB_ERR_ARG;
    const long long warps = (long long)n_tokens * s.H;
    const dim3 grid((unsigned)((warps + 3) / 4));
    const int EW = s.head_form ? s.E + 1 : s.E;
    cudaError_t e;
    if (out_dtype == UB_F32) e = ub_launch_dependent(lin_finish_kernel<float>, grid, dim3(128), 0, st, o, EW, p, s, floor_, w, w_heads, silu_gate, (float*)out, n_tokens, q_scale, eps, out_scale);
    else if (out_dtype == UB_BF16) e = ub_launch_dependent(lin_finish_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, o, EW, p, s, floor_, w, w_heads, silu_gate, (__nv_bfloat16*)out, n_tokens, q_scale, eps, out_scale);
    else return UB_ERR_UNSUPPORTED;
    return (int)e;
}

UB_API int ub_lin_step(const float* p, long long ldp, int n_parts, long long part_stride, const int* shape, const float* up,
                       const float* bias, float tau, const float* bi, const float* bf, float cap, float* S, float* n, float* m,
                       const int* seq_start, const int* seq_slot, const float* w, int w_heads, int silu_gate, void* out,
                       int out_dtype, int n_seqs, float q_scale, float eps, float out_scale, int sm_count, cudaStream_t st) {
    if (n_seqs <= 0) return 0;
    LinShape s;
    if (int rc = read_shape(shape, ldp, n_parts, part_stride, s)) return rc;
    if (n_seqs > 65535) return UB_ERR_ARG;
    if (s.head_form ? (!n || !m || !bi || !bf || !(cap > 0.f)) : (!up || !bias || !(tau > 0.f))) return UB_ERR_ARG;
    StepParams a{p, up, bias, s.head_form ? 0.f : 1.0f / tau, bi, bf, cap, S, n, m, seq_start, seq_slot, w, w_heads, silu_gate, out,
                 q_scale, eps, out_scale};
    const bool vec = s.E % 4 == 0 && ((uintptr_t)S & 15) == 0;
    // blocks that share a head: as many as the SMs hold at once, two each (at least 16 columns a block, and none without any)
    int parts = 1;
    const int width = vec ? 4 : 1;
    auto cols_of = [&](int n) { return ((s.E + n - 1) / n + width - 1) / width * width; };
    while (parts < STEP_PARTS && cols_of(2 * parts) >= 16 && (2 * parts - 1) * cols_of(2 * parts) < s.E &&
           2LL * parts * s.H * n_seqs <= 2LL * (sm_count > 0 ? sm_count : 148)) parts *= 2;
    const int cols = cols_of(parts);
    const int EP = (cols + 3) / 4 * 4;
    const size_t smem = ((size_t)3 * s.D + 4 + 2 * (size_t)EP + (EP > 4 * STEP_THREADS ? EP : 4 * STEP_THREADS)) * sizeof(float);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(parts, s.H, n_seqs);
    cfg.blockDim = dim3(STEP_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = parts;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    static const int plain = [] { const char* v = getenv("ULTIMA_PDL"); return v && v[0] == '0'; }();   // for measurements
    cfg.attrs = attr;
    cfg.numAttrs = plain ? 1 : 2;
    cudaError_t e;
#define GO(TO, VV) e = cudaLaunchKernelEx(&cfg, lin_step_kernel<TO, VV>, a, s, cols)
    if (out_dtype == UB_F32) { if (vec) GO(float, true); else GO(float, false); }
    else if (out_dtype == UB_BF16) { if (vec) GO(__nv_bfloat16, true); else GO(__nv_bfloat16, false); }
    else return UB_ERR_UNSUPPORTED;
#undef GO
    return (int)e;
}
