// Latent attention: a position's keys and values are kept as ONE small vector c (``rank`` numbers, RMS-normed)
// and one rotated key part (``rot`` numbers, possibly none) that all heads share.  A head's unrotated key is W_uk c and its value
// W_uv c; the cache holds only [c | rotated part].  Attention then runs in the latent space: a head's query is
// taken through its own W_uk once (q' = W_uk^T q_unrotated, ``rank`` numbers) so that q' . c = q_unrotated . (W_uk c),
// the score is (q' . c + q_rotated . k_rotated) * scale over ONE shared key row of rank + rot numbers, the
// weighted sum of the rows' leading ``rank`` numbers is taken through W_uv afterwards.  This file holds the
// placement kernel; the two small products a head are batched products (gemm_simt.cu; gemm_tcgen05.cu for bfloat16), the
// attention itself is the ordinary attention over one key head whose value rows are the key rows.
//
// latent_place, from a projection row x (the float32 sum of ``n_parts`` parts), whichever of these has columns there:
//   c_off  [rank | rot] latent columns -> cache row of the position [c / rms(c) * w | rotated key part]
//   d_off  [q_rank] columns of the queries' own latent -> d_out[t] = v / rms(v) * w
//   q_off  the query heads, [dim unrotated | rot rotated] a head ->
//            q_plain[t, h, :dim]          the unrotated query parts, for the product with W_uk^T
//            q_lat[t, h, rank : rank+rot] the rotated query parts (the leading ``rank`` columns are the product's)
//   g_off  [g_width] gate columns -> g_out[t] as they are (float32)
// The rotation turns the pairs (2i, 2i + 1) of the first ``rd`` columns of a rotated part by the position's angles
// (cos, sin [positions, rd / 2], any amplitude already in the tables); other pairings come as a permutation of the weights' rows.
// One block a token for many tokens; for few tokens the sections and the columns are shared out over several blocks a token.
#include "common.cuh"

template <typename TQ, typename TC>
struct LatentPlace {
    long long ldx, part_stride;
    int n_parts;
    int d_off, q_rank; const float* dw; TQ* d_out;
    int q_off; TQ* q_plain; TQ* q_lat;
    int c_off; const float* cw; const float* cs; const float* sn; int rd; TC* kc;
    int g_off, g_width; float* g_out;
    const int* tok_pos; const int* tok_seq;
    int nh, dim, rot, rank;
    float eps;
    int vec;                                         // the query columns four a thread: sizes and places in fours
};

template <typename TX, typename TQ, typename TC>
__global__ void __launch_bounds__(256)
latent_place_kernel(const TX* __restrict__ x, LatentPlace<TQ, TC> p, PagedKV c) {
    extern __shared__ float row[];                   // [max(rank + rot, q_rank)]
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const long long t = blockIdx.x;
    const int tid = threadIdx.x;
    const int pos = p.tok_pos ? p.tok_pos[t] : 0;
    const int half = p.rd >> 1;
    auto at = [&](int col) -> float {
        float v = 0.f;
        for (int s = 0; s < p.n_parts; ++s) v += to_f32<TX>(x[s * p.part_stride + t * p.ldx + col]);
        return v;
    };
    auto turned = [&](float self, float mate, int d) -> float {      // column d of a rotated part; mate: its pair's other column
        const int j = d >> 1;
        const float cj = p.cs[(long long)pos * half + j], sj = p.sn[(long long)pos * half + j];
        return (d & 1) ? self * cj + mate * sj : self * cj - mate * sj;
    };
    if (p.c_off >= 0 && blockIdx.y == 0) {           // the latent columns: the first block of the token's row of blocks
        float ss = 0.f;
        for (int i = tid; i < p.rank + p.rot; i += blockDim.x) {
            const float v = at(p.c_off + i);
            row[i] = v;
            if (i < p.rank) ss += v * v;
        }
        ss = block_sum(ss, red);                      // (also orders the writes of row before the reads below)
        const float inv = inv_rms(ss, (float)p.rank, p.eps);
        TC* dst = p.kc + paged_offset(c, p.tok_seq[t], pos, 0);
        for (int i = tid; i < p.rank + p.rot; i += blockDim.x) {
            float o;
            if (i < p.rank) o = row[i] * inv * p.cw[i];
            else {
                const int d = i - p.rank;
                o = (p.cs && d < p.rd) ? turned(row[i], row[p.rank + (d ^ 1)], d) : row[i];
            }
            dst[i] = from_f32<TC>(o);
        }
        if (gridDim.y == 1) __syncthreads();          // row is used again
    }
    if (p.d_off >= 0 && blockIdx.y == (gridDim.y > 1 ? 1 : 0)) {     // the queries' latent: the second block
        float ss = 0.f;
        for (int i = tid; i < p.q_rank; i += blockDim.x) {
            const float v = at(p.d_off + i);
            row[i] = v;
            ss += v * v;
        }
        const float inv = inv_rms(block_sum(ss, red), (float)p.q_rank, p.eps);
        for (int i = tid; i < p.q_rank; i += blockDim.x) p.d_out[t * p.q_rank + i] = from_f32<TQ>(row[i] * inv * p.dw[i]);
    }
    // the query and gate columns, shared out over the token's blocks
    if (p.q_off >= 0 && p.vec) {                     // four neighbouring columns a thread: both pairs of a rotated part at once
        const int qd = p.dim + p.rot, per = qd >> 2;
        for (int i = blockIdx.y * blockDim.x + tid; i < p.nh * per; i += blockDim.x * gridDim.y) {
            const int h = i / per, d = (i % per) * 4;
            float v[4] = {0.f, 0.f, 0.f, 0.f};
            for (int s = 0; s < p.n_parts; ++s) {
                float a[4];
                load_vec<TX, 4>(x + s * p.part_stride + t * p.ldx + p.q_off + h * qd + d, a);
#pragma unroll
                for (int e = 0; e < 4; ++e) v[e] += a[e];
            }
            if (d < p.dim) { store_vec<TQ, 4>(p.q_plain + (t * p.nh + h) * p.dim + d, v); continue; }
            const int e0 = d - p.dim;
#pragma unroll
            for (int e = 0; e < 4; e += 2)
                if (p.cs && e0 + e < p.rd) {
                    const float u = turned(v[e], v[e + 1], e0 + e), w = turned(v[e + 1], v[e], e0 + e + 1);
                    v[e] = u; v[e + 1] = w;
                }
            store_vec<TQ, 4>(p.q_lat + (t * p.nh + h) * (long long)(p.rank + p.rot) + p.rank + e0, v);
        }
    } else if (p.q_off >= 0) {
        const int qd = p.dim + p.rot;
        for (int i = blockIdx.y * blockDim.x + tid; i < p.nh * qd; i += blockDim.x * gridDim.y) {
            const int h = i / qd, d = i % qd;
            const float v = at(p.q_off + i);
            if (d < p.dim) { p.q_plain[(t * p.nh + h) * p.dim + d] = from_f32<TQ>(v); continue; }
            const int e = d - p.dim;
            float o = v;
            if (p.cs && e < p.rd) o = turned(v, at(p.q_off + h * qd + p.dim + (e ^ 1)), e);
            p.q_lat[(t * p.nh + h) * (long long)(p.rank + p.rot) + p.rank + e] = from_f32<TQ>(o);
        }
    }
    if (p.g_off >= 0)
        for (int i = blockIdx.y * blockDim.x + tid; i < p.g_width; i += blockDim.x * gridDim.y) p.g_out[t * p.g_width + i] = at(p.g_off + i);
}

// Act type and cache type are one (``act_dtype``); offsets below zero leave their section out.
UB_API int ub_latent_place(const void* x, int x_dtype, long long ldx, int n_parts, long long part_stride, int d_off, const float* dw,
                           int q_rank, void* d_out, int q_off, void* q_plain, void* q_lat, int act_dtype, int c_off, const float* cw,
                           const float* cs, const float* sn, int rd, void* kcache, int cache_dtype, int g_off, int g_width,
                           float* g_out, const int* tok_pos, const int* tok_seq, const int* table, int pages_per_seq, int ring,
                           int page, int n_tokens, int nh, int dim, int rot, int rank, float eps, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (n_parts < 1 || rot < 0) return UB_ERR_ARG;
    if (c_off >= 0 && (rank <= 0 || page <= 0 || ring % page != 0 || !cw || !kcache || !table || !tok_pos || !tok_seq)) return UB_ERR_ARG;
    if (d_off >= 0 && (q_rank <= 0 || !dw || !d_out)) return UB_ERR_ARG;
    if (q_off >= 0 && (nh <= 0 || dim <= 0 || !q_plain || !q_lat)) return UB_ERR_ARG;
    if (g_off >= 0 && (g_width <= 0 || !g_out)) return UB_ERR_ARG;
    if (cs && (rd % 2 || rd < 2 || rd > rot || !tok_pos)) return UB_ERR_ARG;
    const int row = max(c_off >= 0 ? rank + rot : 0, d_off >= 0 ? q_rank : 0);
    const size_t smem = (size_t)row * sizeof(float);
    if (smem > 48 * 1024) return UB_ERR_ARG;
    PagedKV c{table, pages_per_seq, ring, page, 1, rank + rot};
    cudaError_t e;
    // for few tokens as many blocks a token as give every thread one query or gate column, up to 16
    const size_t xe = x_dtype == UB_F32 ? 4 : 2, qe = act_dtype == UB_F32 ? 4 : 2;
    const int vec = q_off >= 0 && dim % 4 == 0 && rot % 4 == 0 && rank % 4 == 0 && q_off % 4 == 0 && ldx % 4 == 0 && part_stride % 4 == 0 &&
                    (uintptr_t)x % (4 * xe) == 0 && (uintptr_t)q_plain % (4 * qe) == 0 && (uintptr_t)q_lat % (4 * qe) == 0;
    const int cols = (q_off >= 0 ? nh * (dim + rot) / (vec ? 4 : 1) : 0) + (g_off >= 0 ? g_width : 0);
    const int sections = (c_off >= 0 && d_off >= 0) ? 2 : 1;
    const int per_token = n_tokens > 64 ? 1 : min(16, max(sections, (cols + 255) / 256));
#define GO(TX, TQ) do { \
        const LatentPlace<TQ, TQ> p{ldx, part_stride, n_parts, d_off, q_rank, dw, (TQ*)d_out, q_off, (TQ*)q_plain, (TQ*)q_lat, c_off, cw, \
                                    cs, sn, rd, (TQ*)kcache, g_off, g_width, g_out, tok_pos, tok_seq, nh, dim, rot, rank, eps, vec}; \
        e = ub_launch_dependent(latent_place_kernel<TX, TQ, TQ>, dim3(n_tokens, per_token), dim3(256), smem, st, (const TX*)x, p, c); } while (0)
    if (act_dtype != cache_dtype) return UB_ERR_UNSUPPORTED;
    if (x_dtype == UB_F32 && act_dtype == UB_F32) GO(float, float);
    else if (x_dtype == UB_F32 && act_dtype == UB_BF16) GO(float, __nv_bfloat16);
    else if (x_dtype == UB_BF16 && act_dtype == UB_BF16) GO(__nv_bfloat16, __nv_bfloat16);
    else return UB_ERR_UNSUPPORTED;
#undef GO
    return (int)e;
}
