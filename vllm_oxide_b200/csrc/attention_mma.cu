// Tensor-core attention over the paged cache for the bfloat16 engine: one kernel for portions of
// prompts (and mixed batches), one for steps of single decoded tokens.
//
// Math (as csrc/attention.cu; reference crates/engine/src/backend/cpu/attention.rs:76-128):
//   s_j = (q . K_j) * scale over keys first..p, softmax in float32 with a running maximum,
//   out = sum_j softmax_j V_j. Q K^T and P V run on the tensor cores (mma.sync m16n8k16, bf16 in,
//   float32 accumulate); P is rounded to bfloat16 for the second product; everything between is
//   float32 (exp2 of scores pre-multiplied by scale * log2 e).
//
// Grouped-query packing: the G = H / KV query heads that share a kv head are stacked as rows, so a
// K/V tile is read once per kv head instead of once per head. Row rr of a request's row space is
// token rr / G (position context_len + rr / G) and head kvh * G + rr % G.
//
// K/V tiles of 64 keys are gathered page by page with 16-byte cp.async copies into padded shared
// memory (row stride head_dim + 8 elements keeps ldmatrix free of bank conflicts), double buffered.
// Keys outside [first, p] are never read from global memory (their pages may have been given
// back): their shared-memory rows are zero-filled and their scores masked to -inf.
//
// Kernels take head_dim 64 or 128, page sizes that divide 64, G <= 16 for the decode kernel;
// the launcher refuses anything else (the caller then uses the general kernel).
//
// What may follow the weighted sum (`AttnTail`, all optional): a sink per head (exp(sink) joins the
// softmax's denominator once, a key with no value), a gate (the result times sigmoid(gate[row,
// head * hd + d]), or sigmoid(gate[row, head]) with one number per head) and a constant factor.
#include "common.cuh"
VOB_PDL_SWITCH(attention_mma)

namespace {

constexpr int BN = 64;        // keys per tile
constexpr int NTHREADS = 128;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(smem_u32(dst)), "l"(src));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 2^x by the special-function unit (two units in the last place: far inside what a bfloat16
// probability needs); -inf gives 0.
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
struct AttnTail {
    const float* sink;                // [H], or null
    const __nv_bfloat16* gate;        // [rows, gate_stride], or null
    long long gate_stride;
    float out_scale;
    int gate_heads;                   // the gate has one column per head
};
// The denominator of a row of `head` whose sum `L` is relative to the maximum `Ms` (base-2 scale).
__device__ __forceinline__ float tail_den(const AttnTail& t, int head, float L, float Ms) {
    return t.sink ? L + exp2f(t.sink[head] * 1.4426950408889634f - Ms) : L;
}
__device__ __forceinline__ float tail_val(const AttnTail& t, long long row, int head, int col, float v) {
    v *= t.out_scale;
    if (t.gate) v *= 1.0f / (1.0f + expf(-__bfloat162float(t.gate[row * t.gate_stride + (t.gate_heads ? head : col)])));
    return v;
}

// What may lie between q . k and the softmax (all optional; the kernels built with SHAPED take it):
//   chunk > 0    a query reads only the keys of its own block of `chunk` positions, blocks counted from position 0;
//   a cap        score <- softcap * tanh(score / softcap);
//   r1, r2       [H] each: r1 * ln(1 + r2 * (i - j)) is taken off the score of key j for the query at i.
// Only in the kernels built with KV1 (the values are the cached keys), which take no logarithmic bias and no pooled keys:
//   linear       r1 * (i - j) is taken off (r2 is not used);
//   keep         (with a window) the keys of the first `keep` positions are seen by every query behind them;
//   kscale       one float per cached token (laid out [pages][page_size]): q . k is multiplied by key j's before anything else
//                (the keys' norm, one number per token and a weight per feature, is this number and a factor on q).
// Scores leave in base-2 units (times log2 e), and the launchers' scale_log2 is not used by a shaped kernel. The struct
// is a kernel parameter: what the inner loop reads of it comes from the constant bank and holds no register.
//   pooled keys  (with a window, portion kernel only) beside the window's tokens a query at position p sees the first
//                floor((p + 1 - window) / pool) entries of a second pair of caches, `kp` and `vp`: entry b, stored where a
//                token at position b would be, is the mean key and the mean value of the tokens b * pool .. b * pool + pool - 1.
struct ScoreShape {
    int chunk;
    float pre;            // q . k times this is tanh's argument (scale / softcap); without a cap, the score in base-2 units
    float cap_log2;       // softcap * log2 e, 0: no cap
    const float* r1;
    const float* r2;
    const __nv_bfloat16* kp;      // pooled keys and values (null: none), laid out like the caches
    const __nv_bfloat16* vp;
    int pool;
    int keep;
    int linear;
    const float* kscale;
};
inline ScoreShape make_shape(int chunk, float softcap, const float* r1, const float* r2, float scale, const void* kp = nullptr,
                             const void* vp = nullptr, int pool = 0, int keep = 0, int linear = 0, const float* kscale = nullptr) {
    const float log2e = 1.4426950408889634f;
    return ScoreShape{chunk, softcap > 0.f ? scale / softcap : scale * log2e, softcap > 0.f ? softcap * log2e : 0.f, r1, r2,
                      (const __nv_bfloat16*)kp, (const __nv_bfloat16*)vp, pool, keep, linear, kscale};
}
// The distance bias of a thread's two rows: r1 and r2 of their heads (zero for a row that is no row of the request); a linear
// bias has its slope in base-2 units here.
struct RowShape {
    float r1[2], r2[2];
};
__device__ __forceinline__ RowShape row_shape(const ScoreShape& sh, int head0, int head1) {
    RowShape rs;
    const bool bias = sh.r1 != nullptr;
    rs.r1[0] = bias && head0 >= 0 ? sh.r1[head0] : 0.f;
    rs.r1[1] = bias && head1 >= 0 ? sh.r1[head1] : 0.f;
    if (sh.linear) {
        rs.r1[0] *= 1.4426950408889634f;
        rs.r1[1] *= 1.4426950408889634f;
    }
    rs.r2[0] = bias && !sh.linear && head0 >= 0 ? sh.r2[head0] : 0.f;
    rs.r2[1] = bias && !sh.linear && head1 >= 0 ? sh.r2[head1] : 0.f;
    return rs;
}
// The first key a query at `pos` reads (0 for a row of position -1, which is no row of a request).
__device__ __forceinline__ int first_key(int pos, int window, int chunk) {
    int lo = window > 0 ? max(0, pos + 1 - window) : 0;
    return chunk > 0 ? max(lo, pos - pos % chunk) : lo;
}
// tanh from one exponential and one division: absolute error of a few 1e-7 (the argument is clamped where
// tanh is 1 to float32's last place), which a capped score of some tens keeps far below one bfloat16 step of q . k.
__device__ __forceinline__ float fast_tanh(float x) {
    x = fminf(fmaxf(x, -15.f), 15.f);
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * 2.885390081777927f));
    return 1.f - __fdividef(2.f, e + 1.f);
}

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

// Gather one tile of 64 keys (K and V of one kv head) into shared memory. Keys outside
// [lo, hi) and [0, keep) are zero-filled and never touched in global memory.
// VALUES false: only K. Page numbers come from `s_pages`,
// this block's copy of its request's block-table entries starting at logical page `page0` (a
// global lookup per key would put a dependent L2 round trip in front of every copy); page sizes
// are powers of two (they divide 64), so positions split into page and offset by shift and mask.
template <int HD, bool VALUES = true>
__device__ __forceinline__ void load_kv_tile(__nv_bfloat16* sK, __nv_bfloat16* sV, const __nv_bfloat16* __restrict__ kc,
                                             const __nv_bfloat16* __restrict__ vc, const int* s_pages, int page0, int kvh,
                                             int KV, int page_shift, int tile_start, int lo, int hi, int keep = 0) {
    constexpr int LD = HD + 8;
    constexpr int CH = HD / 8;                 // 16-byte pieces per key
    constexpr int KEYS_PER_PASS = NTHREADS / CH;
    const int ch = threadIdx.x % CH;
    const int k0 = threadIdx.x / CH;
    const int page_size = 1 << page_shift;
#pragma unroll
    for (int key = k0; key < BN; key += KEYS_PER_PASS) {
        int j = tile_start + key;
        __nv_bfloat16* dk = sK + key * LD + ch * 8;
        __nv_bfloat16* dv = sV + key * LD + ch * 8;
        if ((j >= lo || j < keep) && j < hi) {
            int page = s_pages[(j >> page_shift) - page0];
            size_t off = ((((size_t)page * KV + kvh) << page_shift) + (j & (page_size - 1))) * HD + ch * 8;
            cp_async16(dk, kc + off);
            if (VALUES) cp_async16(dv, vc + off);
        } else {
            *reinterpret_cast<uint4*>(dk) = make_uint4(0, 0, 0, 0);
            if (VALUES) *reinterpret_cast<uint4*>(dv) = make_uint4(0, 0, 0, 0);
        }
    }
}

// The tile's 64 numbers per cached token (ones without `kscale`) into shared memory, for the same keys.
__device__ __forceinline__ void load_key_scales(float* sR, const float* __restrict__ kscale, const int* s_pages, int page0, int page_shift,
                                                int tile_start, int lo, int hi, int keep) {
    if (threadIdx.x >= BN) return;
    const int j = tile_start + threadIdx.x;
    float* d = sR + threadIdx.x;
    if (kscale && (j >= lo || j < keep) && j < hi) {
        const float* s = kscale + ((size_t)s_pages[(j >> page_shift) - page0] << page_shift) + (j & ((1 << page_shift) - 1));
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(smem_u32(d)), "l"(s));
    } else {
        *d = 1.f;
    }
}

// S (16 rows x 8*NB keys) += Q K^T for the n-blocks [nb0, nb0+NB) of the tile in sK.
template <int HD, int NB>
__device__ __forceinline__ void qk_tile(float (&s)[NB][4], const uint32_t (&qf)[HD / 16][4], const __nv_bfloat16* sK, int nb0) {
    constexpr int LD = HD + 8;
    int lane = threadIdx.x & 31;
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
#pragma unroll
        for (int i = 0; i < 4; ++i) s[nb][i] = 0.f;
#pragma unroll
        for (int k2 = 0; k2 < HD / 32; ++k2) {
            uint32_t r[4];
            ldmatrix_x4(r, sK + ((nb0 + nb) * 8 + (lane & 7)) * LD + k2 * 32 + (lane >> 3) * 8);
            mma_bf16(s[nb], qf[2 * k2], r[0], r[1]);
            mma_bf16(s[nb], qf[2 * k2 + 1], r[2], r[3]);
        }
    }
}

// O (16 x HD) += P V for NK slices of 16 keys starting at key slice ks0 of the tile in sV.
template <int HD, int NK>
__device__ __forceinline__ void pv_tile(float (&o)[HD / 8][4], const uint32_t (&pa)[NK][4], const __nv_bfloat16* sV, int ks0) {
    constexpr int LD = HD + 8;
    int lane = threadIdx.x & 31;
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
#pragma unroll
        for (int n2 = 0; n2 < HD / 16; ++n2) {
            uint32_t r[4];
            ldmatrix_x4_trans(r, sV + ((ks0 + kk) * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + n2 * 16 + (lane >> 4) * 8);
            mma_bf16(o[2 * n2], pa[kk], r[0], r[1]);
            mma_bf16(o[2 * n2 + 1], pa[kk], r[2], r[3]);
        }
    }
}

// Mask, running maximum, exponentials; returns P as A-fragments. s holds NB n-blocks of 8 keys
// starting at key index key0; this thread's rows are r and r+8 with limits [lo, pos]. With MASK
// false the caller knows that every key of the tile is visible to every row of the warp. SHAPED: the scores
// first become what `rs` makes of them (cap, distance bias), in base-2 units, and `scale_log2` is not used.
// KV1: q . k is first multiplied by key j's number, ksc[j - key0]; the distance bias is the linear one (a slope of 0: none), and
// keys of kept first tokens are seen too.
template <int NB, int HDN, bool MASK, bool SHAPED = false, bool KV1 = false>
__device__ __forceinline__ void softmax_step(float (&s)[NB][4], uint32_t (&pa)[NB / 2][4], float (&o)[HDN][4],
                                             float (&m)[2], float (&l)[2], int key0, const int (&lo)[2],
                                             const int (&pos)[2], float scale_log2, const ScoreShape* sh = nullptr,
                                             const RowShape* rs = nullptr, const float* ksc = nullptr) {
    int lane = threadIdx.x & 31;
    float mx[2] = {-INFINITY, -INFINITY};
    if (SHAPED) scale_log2 = 1.f;
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            int h = i >> 1;
            if (SHAPED) {
                int j = key0 + nb * 8 + (lane & 3) * 2 + (i & 1);
                float t = s[nb][i] * sh->pre;
                if (KV1) t *= ksc[nb * 8 + (lane & 3) * 2 + (i & 1)];
                if (sh->cap_log2 > 0.f) t = sh->cap_log2 * fast_tanh(t);
                if (KV1) t = fmaf(-rs->r1[h], (float)(pos[h] - j), t);
                else if (sh->r1) t -= rs->r1[h] * __log2f(fmaf(rs->r2[h], (float)max(pos[h] - j, 0), 1.f));
                s[nb][i] = t;
            }
            if (MASK) {
                int j = key0 + nb * 8 + (lane & 3) * 2 + (i & 1);
                if (!((j >= lo[h] || (KV1 && j < sh->keep)) && j <= pos[h])) s[nb][i] = -INFINITY;
            }
            mx[h] = fmaxf(mx[h], s[nb][i]);
        }
    }
    float alpha[2], msafe[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
        float mn = fmaxf(m[h], mx[h] * scale_log2);   // scale > 0: the maximum of the scaled scores
        msafe[h] = mn == -INFINITY ? 0.f : mn;
        alpha[h] = fast_exp2(m[h] - msafe[h]);         // m = -inf: 0
        m[h] = mn;
        l[h] *= alpha[h];
    }
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float p = fast_exp2(fmaf(s[nb][i], scale_log2, -msafe[i >> 1]));
            s[nb][i] = p;
            l[i >> 1] += p;                           // this thread's share; the quad is summed at the end
        }
    }
#pragma unroll
    for (int n = 0; n < HDN; ++n) {
        o[n][0] *= alpha[0]; o[n][1] *= alpha[0];
        o[n][2] *= alpha[1]; o[n][3] *= alpha[1];
    }
#pragma unroll
    for (int kk = 0; kk < NB / 2; ++kk) {
        pa[kk][0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
        pa[kk][1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
        pa[kk][2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
        pa[kk][3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
    }
}

// ---------------------------------------------------------------------------------------------
// Portions of prompts and mixed batches. Grid (row tiles, requests, kv heads); a block of 4 warps
// owns 64 rows of one request's row space (16 rows per warp) and walks the key tiles that any of
// its rows can see. Blocks beyond a request's rows leave at once.
// Bound: tensor-core and exp throughput for long portions; for short ones the K/V reads.
// ---------------------------------------------------------------------------------------------
template <int HD>
__global__ void __launch_bounds__(NTHREADS)
attn_prefill_mma_kernel(const __nv_bfloat16* __restrict__ q, long long q_stride, __nv_bfloat16* __restrict__ out,
                        long long out_stride, const __nv_bfloat16* __restrict__ kc, const __nv_bfloat16* __restrict__ vc,
                        const int* __restrict__ block_tables, int max_pages, const int* __restrict__ seq_starts,
                        const int* __restrict__ context_lens, int H, int KV, int page_shift, int window, float scale_log2,
                        AttnTail tail) {
    constexpr int LD = HD + 8;
    constexpr int BM = 64;
    pdl_launch_dependents();
    pdl_wait(7);
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* sK0 = sQ + BM * LD;
    __nv_bfloat16* sV0 = sK0 + 2 * BN * LD;
    int* s_pages = reinterpret_cast<int*>(sV0 + 2 * BN * LD);            // [max_pages]

    const int G = H / KV;
    // Blocks are handed out in the order x, y, z: the kv head runs fastest and the row tile slowest,
    // later row tiles (which see more keys) first, so that over the whole grid the long blocks
    // start first and the short ones fill the gaps behind them.
    const int kvh = blockIdx.x, seq = blockIdx.y;
    const int row0 = seq_starts[seq];
    const int n_new = seq_starts[seq + 1] - row0;
    const int total_rows = n_new * G;
    const int tile_row0 = (gridDim.z - 1 - blockIdx.z) * BM;
    if (tile_row0 >= total_rows) return;
    const int ctx = context_lens[seq];
    const int* bt = block_tables + (size_t)seq * max_pages;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    // rows of this block -> shared memory (zero for rows beyond the request)
    for (int c = threadIdx.x; c < BM * (HD / 8); c += NTHREADS) {
        int r = c / (HD / 8), ch = c - r * (HD / 8);
        int rr = tile_row0 + r;
        __nv_bfloat16* dst = sQ + r * LD + ch * 8;
        if (rr < total_rows) {
            int tok = rr / G, head = kvh * G + rr % G;
            cp_async16(dst, q + (size_t)(row0 + tok) * q_stride + (size_t)head * HD + ch * 8);
        } else {
            *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
    }
    // key range any row of the block reads
    const int last_rr = min(tile_row0 + BM, total_rows) - 1;
    const int hi = ctx + last_rr / G + 1;
    const int first_tok_pos = ctx + tile_row0 / G;
    const int lo_blk = window > 0 ? max(0, first_tok_pos + 1 - window) : 0;
    const int t_begin = lo_blk / BN, t_end = (hi + BN - 1) / BN;
    // this block's pages: logical pages [page0, page_end) of the request, one coalesced read
    const int page0 = lo_blk >> page_shift, page_end = ((hi - 1) >> page_shift) + 1;
    for (int i = threadIdx.x; i < page_end - page0; i += NTHREADS) s_pages[i] = bt[page0 + i];
    __syncthreads();

    load_kv_tile<HD>(sK0, sV0, kc, vc, s_pages, page0, kvh, KV, page_shift, t_begin * BN, lo_blk, hi);
    cp_async_commit();

    int pos[2], lo[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        int rr = tile_row0 + warp * 16 + (lane >> 2) + h * 8;
        pos[h] = rr < total_rows ? ctx + rr / G : -1;
        lo[h] = window > 0 ? max(0, pos[h] + 1 - window) : 0;
    }
    // the warp's position range: tiles beyond its last position are skipped, tiles wholly inside
    // every row's [lo, pos] need no mask (rows beyond the request count as position -1: masked)
    int warp_last_pos = max(pos[0], pos[1]), warp_first_pos = min(pos[0], pos[1]), warp_max_lo = max(lo[0], lo[1]);
#pragma unroll
    for (int x = 4; x < 32; x <<= 1) {
        warp_last_pos = max(warp_last_pos, __shfl_xor_sync(0xffffffffu, warp_last_pos, x));
        warp_first_pos = min(warp_first_pos, __shfl_xor_sync(0xffffffffu, warp_first_pos, x));
        warp_max_lo = max(warp_max_lo, __shfl_xor_sync(0xffffffffu, warp_max_lo, x));
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    float o[HD / 8][4];
#pragma unroll
    for (int n = 0; n < HD / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.f;
    uint32_t qf[HD / 16][4];

    for (int t = t_begin; t < t_end; ++t) {
        int buf = (t - t_begin) & 1;
        __nv_bfloat16* sK = sK0 + buf * BN * LD;
        __nv_bfloat16* sV = sV0 + buf * BN * LD;
        cp_async_wait<0>();
        __syncthreads();                       // tile t (and Q) visible; everyone is done with tile t-1
        if (t + 1 < t_end) {
            load_kv_tile<HD>(sK0 + (buf ^ 1) * BN * LD, sV0 + (buf ^ 1) * BN * LD, kc, vc, s_pages, page0, kvh, KV, page_shift,
                             (t + 1) * BN, lo_blk, hi);
            cp_async_commit();
        }
        if (t == t_begin) {
#pragma unroll
            for (int kk = 0; kk < HD / 16; ++kk)
                ldmatrix_x4(qf[kk], sQ + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + kk * 16 + (lane >> 4) * 8);
        }
        // a warp whose rows all lie before this tile's first key has nothing to do here
        if (t * BN <= warp_last_pos) {
            float s[8][4];
            qk_tile<HD, 8>(s, qf, sK, 0);
            uint32_t pa[4][4];
            // no masking where the whole tile lies inside [lo, pos] of every row of the warp
            if ((t + 1) * BN - 1 <= warp_first_pos && t * BN >= warp_max_lo)
                softmax_step<8, HD / 8, false>(s, pa, o, m, l, t * BN, lo, pos, scale_log2);
            else
                softmax_step<8, HD / 8, true>(s, pa, o, m, l, t * BN, lo, pos, scale_log2);
            pv_tile<HD, 4>(o, pa, sV, 0);
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        int rr = tile_row0 + warp * 16 + (lane >> 2) + h * 8;
        if (rr >= total_rows) continue;
        int tok = rr / G, head = kvh * G + rr % G;
        float inv = 1.0f / tail_den(tail, head, l[h], m[h]);
        __nv_bfloat16* op = out + (size_t)(row0 + tok) * out_stride + (size_t)head * HD + (lane & 3) * 2;
        const int col = head * HD + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < HD / 8; ++n)
            *reinterpret_cast<uint32_t*>(op + n * 8) = pack_bf16(tail_val(tail, row0 + tok, head, col + n * 8, o[n][2 * h] * inv),
                                                                 tail_val(tail, row0 + tok, head, col + n * 8 + 1, o[n][2 * h + 1] * inv));
    }
}

// ---------------------------------------------------------------------------------------------
// The same for keys of D and values of DV features (multiples of 8 up to 128, different or not): the tiles in
// shared memory are HD = D rounded up to a multiple of 32 and HDV = DV rounded up to 32, 64 or 128 wide, the
// columns beyond the real sizes zero (a zero column of Q and K adds nothing to a score, a zero column of V
// gives an output column that is not stored). Same grid, same walk over the key tiles, same tail. KV1: the values are the
// cached keys (HDV == HD): a tile is fetched once and serves both products, with a number per key beside it (`ScoreShape`).
// ---------------------------------------------------------------------------------------------
template <int W>
__device__ __forceinline__ void load_rows_padded(__nv_bfloat16* dst, const __nv_bfloat16* __restrict__ cache, int real, const int* s_pages,
                                                 int page0, int kvh, int KV, int page_shift, int tile_start, int lo, int hi, int keep = 0) {
    constexpr int LD = W + 8, CH = W / 8;
    const int page_size = 1 << page_shift, real_ch = real >> 3;
    for (int idx = threadIdx.x; idx < BN * CH; idx += NTHREADS) {
        const int key = idx / CH, ch = idx - key * CH;
        const int j = tile_start + key;
        __nv_bfloat16* d = dst + key * LD + ch * 8;
        if (ch < real_ch && (j >= lo || j < keep) && j < hi) {
            const int page = s_pages[(j >> page_shift) - page0];
            cp_async16(d, cache + ((((size_t)page * KV + kvh) << page_shift) + (j & (page_size - 1))) * real + ch * 8);
        } else {
            *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
        }
    }
}

// Blocks per SM the compiler is told to aim at, where its own choice of registers would spill a few bytes (0: its own choice).
constexpr int any_min_blocks(int hd, int hdv, bool shaped, bool kv1) {
    return shaped && !kv1 && hd == 32 && hdv == 32 ? 3 : 0;
}
template <int HD, int HDV, bool SHAPED, bool KV1>
__global__ void __launch_bounds__(NTHREADS, any_min_blocks(HD, HDV, SHAPED, KV1))
attn_prefill_mma_any_kernel(const __nv_bfloat16* __restrict__ q, long long q_stride, __nv_bfloat16* __restrict__ out,
                            long long out_stride, const __nv_bfloat16* __restrict__ kc, const __nv_bfloat16* __restrict__ vc,
                            const int* __restrict__ block_tables, int max_pages, const int* __restrict__ seq_starts,
                            const int* __restrict__ context_lens, int H, int KV, int D, int DV, int page_shift, int window,
                            float scale_log2, AttnTail tail, ScoreShape shape) {
    constexpr int LD = HD + 8, LDV = HDV + 8;
    constexpr int BM = 64;
    pdl_launch_dependents();
    pdl_wait(9);
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* sK0 = sQ + BM * LD;
    static_assert(!KV1 || (SHAPED && HD == HDV), "one tile serves both products");
    __nv_bfloat16* sV0 = KV1 ? sK0 : sK0 + 2 * BN * LD;
    float* sR0 = reinterpret_cast<float*>(sK0 + 2 * BN * LD);            // KV1: [2][BN] a number per key
    // [2 * max_pages]: the tokens' pages, then the kept first tokens' or the pooled entries'
    int* s_pages = KV1 ? reinterpret_cast<int*>(sR0 + 2 * BN) : reinterpret_cast<int*>(sV0 + 2 * BN * LDV);

    const int G = H / KV;
    const int kvh = blockIdx.x, seq = blockIdx.y;
    const int row0 = seq_starts[seq];
    const int n_new = seq_starts[seq + 1] - row0;
    const int total_rows = n_new * G;
    const int tile_row0 = (gridDim.z - 1 - blockIdx.z) * BM;
    if (tile_row0 >= total_rows) return;
    const int ctx = context_lens[seq];
    const int* bt = block_tables + (size_t)seq * max_pages;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    for (int c = threadIdx.x; c < BM * (HD / 8); c += NTHREADS) {
        int r = c / (HD / 8), ch = c - r * (HD / 8);
        int rr = tile_row0 + r;
        __nv_bfloat16* dst = sQ + r * LD + ch * 8;
        if (rr < total_rows && ch * 8 < D) {
            int tok = rr / G, head = kvh * G + rr % G;
            cp_async16(dst, q + (size_t)(row0 + tok) * q_stride + (size_t)head * D + ch * 8);
        } else {
            *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
    }
    const int last_rr = min(tile_row0 + BM, total_rows) - 1;
    const int hi = ctx + last_rr / G + 1;
    const int first_tok_pos = ctx + tile_row0 / G;
    const int chunk = SHAPED ? shape.chunk : 0;
    const int lo_blk = first_key(first_tok_pos, window, chunk);      // the block's first row reads furthest back
    const int pool = SHAPED && !KV1 && shape.kp ? shape.pool : 0;
    // pooled entries the block's last row sees (the most of all its rows)
    const int hi_pool = pool > 0 && window > 0 && hi - window >= pool ? (hi - window) / pool : 0;

    int pos[2], lo[2], hd[2], pos_p[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        int rr = tile_row0 + warp * 16 + (lane >> 2) + h * 8;
        pos[h] = rr < total_rows ? ctx + rr / G : -1;
        hd[h] = rr < total_rows ? kvh * G + rr % G : -1;
        lo[h] = first_key(pos[h], window, chunk);
        // the last pooled entry this row sees (-1: none)
        pos_p[h] = pool > 0 && pos[h] >= 0 && pos[h] + 1 - window >= pool ? (pos[h] + 1 - window) / pool - 1 : -1;
    }
    RowShape rs;
    if (SHAPED) rs = row_shape(shape, hd[0], hd[1]);
    int warp_last_pos = max(pos[0], pos[1]), warp_first_pos = min(pos[0], pos[1]), warp_max_lo = max(lo[0], lo[1]);
    int warp_min_lo = 0;                             // blocks of positions: the first key any row of the warp reads
    if (SHAPED) warp_min_lo = min(pos[0] < 0 ? 0x7fffffff : lo[0], pos[1] < 0 ? 0x7fffffff : lo[1]);
    int warp_last_p = max(pos_p[0], pos_p[1]), warp_first_p = min(pos_p[0], pos_p[1]);
#pragma unroll
    for (int x = 4; x < 32; x <<= 1) {
        warp_last_pos = max(warp_last_pos, __shfl_xor_sync(0xffffffffu, warp_last_pos, x));
        warp_first_pos = min(warp_first_pos, __shfl_xor_sync(0xffffffffu, warp_first_pos, x));
        warp_max_lo = max(warp_max_lo, __shfl_xor_sync(0xffffffffu, warp_max_lo, x));
        if (SHAPED && !KV1) warp_last_p = max(warp_last_p, __shfl_xor_sync(0xffffffffu, warp_last_p, x));
        if (SHAPED && !KV1) warp_first_p = min(warp_first_p, __shfl_xor_sync(0xffffffffu, warp_first_p, x));
        if (SHAPED) warp_min_lo = min(warp_min_lo, __shfl_xor_sync(0xffffffffu, warp_min_lo, x));
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    float o[HDV / 8][4];
#pragma unroll
    for (int n = 0; n < HDV / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.f;
    uint32_t qf[HD / 16][4];
    // One walk over key tiles with one running softmax: first the tiles of pooled entries or of kept first tokens (where
    // there are any, and not the tiles the window reaches itself), then the tiles of tokens. Both page lists sit in shared
    // memory, the tokens' first.
    const int t_begin = lo_blk / BN, t_end = (hi + BN - 1) / BN;
    const int keep = KV1 ? shape.keep : 0;
    const int tp_end = KV1 ? min((keep + BN - 1) / BN, t_begin) : (hi_pool + BN - 1) / BN;
    const int page0 = (t_begin * BN) >> page_shift, page_end = ((hi - 1) >> page_shift) + 1;
    int* s_pages_p = s_pages + (page_end - page0);
    const int pages_p = KV1 ? (tp_end * BN) >> page_shift : hi_pool > 0 ? ((hi_pool - 1) >> page_shift) + 1 : 0;
    for (int i = threadIdx.x; i < page_end - page0 + pages_p; i += NTHREADS) s_pages[i] = i < page_end - page0 ? bt[page0 + i] : bt[i - (page_end - page0)];
    __syncthreads();
    const int n_it = tp_end + (t_end - t_begin);
    auto load_tile = [&](int it, int buf) {
        if (KV1) {
            const bool kept = it < tp_end;
            const int t = kept ? it : t_begin + it - tp_end, lo_t = kept ? 0 : lo_blk, hi_t = kept ? keep : hi, p0 = kept ? 0 : page0;
            const int* pages = kept ? s_pages_p : s_pages;
            load_rows_padded<HD>(sK0 + buf * BN * LD, kc, D, pages, p0, kvh, KV, page_shift, t * BN, lo_t, hi_t, keep);
            load_key_scales(sR0 + buf * BN, shape.kscale, pages, p0, page_shift, t * BN, lo_t, hi_t, keep);
        } else if (SHAPED && it < tp_end) {
            load_rows_padded<HD>(sK0 + buf * BN * LD, shape.kp, D, s_pages_p, 0, kvh, KV, page_shift, it * BN, 0, hi_pool);
            load_rows_padded<HDV>(sV0 + buf * BN * LDV, shape.vp, DV, s_pages_p, 0, kvh, KV, page_shift, it * BN, 0, hi_pool);
        } else {
            const int t = t_begin + it - tp_end;
            load_rows_padded<HD>(sK0 + buf * BN * LD, kc, D, s_pages, page0, kvh, KV, page_shift, t * BN, lo_blk, hi);
            load_rows_padded<HDV>(sV0 + buf * BN * LDV, vc, DV, s_pages, page0, kvh, KV, page_shift, t * BN, lo_blk, hi);
        }
        cp_async_commit();
    };
    load_tile(0, 0);
    for (int it = 0; it < n_it; ++it) {
        const int buf = it & 1;
        __nv_bfloat16* sK = sK0 + buf * BN * LD;
        __nv_bfloat16* sV = sV0 + buf * BN * LDV;
        cp_async_wait<0>();
        __syncthreads();                       // this tile (and Q) visible; everyone is done with the tile before
        if (it + 1 < n_it) load_tile(it + 1, buf ^ 1);
        if (it == 0) {
#pragma unroll
            for (int kk = 0; kk < HD / 16; ++kk)
                ldmatrix_x4(qf[kk], sQ + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + kk * 16 + (lane >> 4) * 8);
        }
        const bool pooled = SHAPED && !KV1 && it < tp_end;
        const int t = SHAPED && it < tp_end ? it : t_begin + it - tp_end;
        const int w_last = pooled ? warp_last_p : warp_last_pos, w_first = pooled ? warp_first_p : warp_first_pos;
        const int w_max_lo = pooled ? 0 : warp_max_lo, w_min_lo = pooled ? 0 : warp_min_lo;
        const int lo_r[2] = {pooled ? 0 : lo[0], pooled ? 0 : lo[1]}, pos_r[2] = {pooled ? pos_p[0] : pos[0], pooled ? pos_p[1] : pos[1]};
        // a tile behind the warp's last key needs no work, nor has one whose rows all begin to read behind this tile's last key
        // (unless it holds kept first tokens)
        if (t * BN <= w_last && (!SHAPED || (t + 1) * BN > w_min_lo || (KV1 && t * BN < keep))) {
            float s[8][4];
            qk_tile<HD, 8>(s, qf, sK, 0);
            uint32_t pa[4][4];
            const float* ksc = sR0 + buf * BN;
            if ((t + 1) * BN - 1 <= w_first && (t * BN >= w_max_lo || (KV1 && (t + 1) * BN <= keep)))
                softmax_step<8, HDV / 8, false, SHAPED, KV1>(s, pa, o, m, l, t * BN, lo_r, pos_r, scale_log2, &shape, &rs, ksc);
            else
                softmax_step<8, HDV / 8, true, SHAPED, KV1>(s, pa, o, m, l, t * BN, lo_r, pos_r, scale_log2, &shape, &rs, ksc);
            pv_tile<HDV, 4>(o, pa, sV, 0);
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        int rr = tile_row0 + warp * 16 + (lane >> 2) + h * 8;
        if (rr >= total_rows) continue;
        int tok = rr / G, head = kvh * G + rr % G;
        float inv = 1.0f / tail_den(tail, head, l[h], m[h]);
        __nv_bfloat16* op = out + (size_t)(row0 + tok) * out_stride + (size_t)head * DV + (lane & 3) * 2;
        const int col = head * DV + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < HDV / 8; ++n)
            if (n * 8 + (lane & 3) * 2 < DV)
                *reinterpret_cast<uint32_t*>(op + n * 8) = pack_bf16(tail_val(tail, row0 + tok, head, col + n * 8, o[n][2 * h] * inv),
                                                                     tail_val(tail, row0 + tok, head, col + n * 8 + 1, o[n][2 * h + 1] * inv));
    }
}

constexpr int DEC_MIN_TILES = 3;            // measured on whole decode steps at batch 1: 8,192 keys 0.808 ms with 3, 0.838 with 2, 0.812 with 4
constexpr int DEC_MAX_SPLITS_WIDE = 64;

// The block of a request and kv head that arrives last adds the partials of all `splits` blocks
// up (merge through global memory). Everything is fetched with independent loads: first every
// partial's maxima and sums, from which each row's weights follow; then the values, a thread
// taking four neighbouring dims over one half of the partials, in rank order. `scratch` is the
// block's shared memory behind q; `out` points at the group's first head. Not inlined: the
// kernel's main path keeps its registers.
template <int HD>
__device__ __noinline__ void merge_partials(const float* __restrict__ all, int splits, int G, float* scratch,
                                            __nv_bfloat16* __restrict__ out, const AttnTail& tail, int row, int head0) {
    constexpr int PART = 16 * HD + 32;
    float* ml = scratch;                                    // [splits][32]: 16 maxima, 16 sums
    float* fk = ml + DEC_MAX_SPLITS_WIDE * 32;              // [splits][16]: weight of partial k in row r
    float* hs = fk + DEC_MAX_SPLITS_WIDE * 16;              // [2][16 * HD]: the two halves' sums
    float* Lrow = hs + 2 * 16 * HD;                         // [16]
    static_assert(DEC_MAX_SPLITS_WIDE * 48 + 2 * 16 * HD + 16 <= 128 + 4 * 16 * HD + 16 * HD + 32, "merge scratch exceeds the combine area");
    for (int i = threadIdx.x; i < splits * 32; i += NTHREADS) ml[i] = __ldcg(all + (size_t)(i >> 5) * PART + 16 * HD + (i & 31));
    __syncthreads();
    if (threadIdx.x < G) {
        const int r = threadIdx.x;
        float M = -INFINITY;
        for (int k = 0; k < splits; ++k) M = fmaxf(M, ml[k * 32 + r]);
        const float Ms = M == -INFINITY ? 0.f : M;
        float L = 0.f;
        for (int k = 0; k < splits; ++k) {
            const float f = exp2f(ml[k * 32 + r] - Ms);
            fk[k * 16 + r] = f;
            L += f * ml[k * 32 + 16 + r];
        }
        Lrow[r] = tail_den(tail, head0 + r, L, Ms);
    }
    __syncthreads();
    const int items = G * HD / 4, k_half = splits / 2;
    for (int it = threadIdx.x; it < 2 * items; it += NTHREADS) {
        const int second = it >= items, e = (it - second * items) * 4, r = e / HD;
        const int k0 = second ? k_half : 0, k1 = second ? splits : k_half;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int k = k0; k < k1; ++k) {
            const float4 v = __ldcg(reinterpret_cast<const float4*>(all + (size_t)k * PART + e));
            const float f = fk[k * 16 + r];
            acc.x += f * v.x; acc.y += f * v.y; acc.z += f * v.z; acc.w += f * v.w;
        }
        *reinterpret_cast<float4*>(hs + second * 16 * HD + e) = acc;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < G * HD; e += NTHREADS) {
        const float L = Lrow[e / HD];
        out[e] = __float2bfloat16_rn(L > 0.f ? tail_val(tail, row, head0 + e / HD, head0 * HD + e, (hs[e] + hs[16 * HD + e]) / L) : 0.f);
    }
}

// ---------------------------------------------------------------------------------------------
// Steps of single decoded tokens. Grid (requests, kv heads, splits): a block reads its share of
// the request's key tiles once for all G heads of the group; its 4 warps split every tile's 64
// keys (16 each) and combine through shared memory. The `splits` blocks of one (request, kv
// head) form a thread-block cluster: every block finishes a share of the outputs, and each sends
// the pieces of its unnormalised partial (running maximum, sum, weighted values) to the blocks
// that finish them, by stores into their shared memory (a region that nothing else uses, so a
// fast peer may write while the owner still works on its tiles); the cluster meets at a barrier
// once, and every block then adds up what it was sent in rank order (a fixed order, so the result
// does not depend on timing) and leaves: nobody reads a peer's memory, so nobody has to wait for
// the others to finish. K/V tiles go
// through a cp.async ring of three stages (two when the grid is so large that the smaller
// footprint lets one more block live on an SM). Bound: the K/V reads (memory).
//
// Few requests with long contexts would leave most SMs idle with 8 blocks each. For them the
// grid has up to 64 splits and no cluster (`partials` is given): a request uses as many of its
// blocks as it has tiles for (at least DEC_MIN_TILES each; the others leave at once), every
// block writes its partial to global memory and counts itself in, and the block that arrives
// last adds the partials up in rank order and puts the counter back to zero. Nobody waits.
// ---------------------------------------------------------------------------------------------

// Shared memory of a decode block: the K/V ring (used again for the combine of the four warps),
// then what the cluster's peers send, then the block's page list.
template <int HD, int DEC_STAGES, bool KV1> __host__ __device__ constexpr size_t decode_ring_bytes() {
    size_t ring = (size_t)(16 + (KV1 ? 1 : 2) * DEC_STAGES * BN) * (HD + 8) * sizeof(__nv_bfloat16) + (KV1 ? DEC_STAGES * BN * sizeof(float) : 0);
    size_t combine = 16 * (HD + 8) * sizeof(__nv_bfloat16) + (size_t)(128 + 4 * 16 * HD + 16 * HD + 32) * sizeof(float);
    return ((ring > combine ? ring : combine) + 15) / 16 * 16;
}
__host__ __device__ constexpr size_t decode_recv_bytes(int G, int HD) { return (size_t)(G * HD + 8 + 256) * sizeof(float); }

// KV1: the values are the cached keys; the ring holds one tile a stage, which serves both products, and a number per key.
// Kept first tokens (ScoreShape::keep): their tiles come first in a request's list of tiles, in front of the window's.
template <int HD, int DEC_STAGES, bool SHAPED, bool KV1>
__global__ void __launch_bounds__(NTHREADS)
attn_decode_mma_kernel(const __nv_bfloat16* __restrict__ q, long long q_stride, __nv_bfloat16* __restrict__ out,
                       long long out_stride, const __nv_bfloat16* __restrict__ kc, const __nv_bfloat16* __restrict__ vc,
                       const int* __restrict__ block_tables, int max_pages, const int* __restrict__ positions,
                       int H, int KV, int page_shift, int window, float scale_log2, float* __restrict__ partials,
                       int* __restrict__ arrived, AttnTail tail, ScoreShape shape) {
    constexpr int LD = HD + 8;
    constexpr int PART = 16 * HD + 32;                                          // floats of one block's partial
    pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ int s_last;
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem_raw);            // 16 x LD
    __nv_bfloat16* sK0 = sQ + 16 * LD;                                          // DEC_STAGES x BN x LD
    __nv_bfloat16* sV0 = KV1 ? sK0 : sK0 + DEC_STAGES * BN * LD;
    float* sR0 = reinterpret_cast<float*>(sK0 + DEC_STAGES * BN * LD);          // KV1: DEC_STAGES x BN numbers
    // what the peers of a cluster send this block: [splits][chunk] values, [8][16] maxima, [8][16] sums
    float* recv_val = reinterpret_cast<float*>(smem_raw + decode_ring_bytes<HD, DEC_STAGES, KV1>());
    float* recv_m = recv_val + (H / KV) * HD + 8;
    float* recv_l = recv_m + 128;
    // this block's pages (a launch without a cluster has no region for what peers send)
    int* s_pages = (!partials && gridDim.z > 1) ? reinterpret_cast<int*>(recv_l + 128) : reinterpret_cast<int*>(recv_val);

    // Positions and block tables were put on the device before this step's kernels began, and
    // every key but the newest was written by earlier steps: all of that may be read before the
    // wait, while the kernel in front (which writes the newest key and this step's q) still runs.
    const int G = H / KV;
    const int seq = blockIdx.x, kvh = blockIdx.y, split = blockIdx.z;
    int splits = gridDim.z;
    // every block of the cluster has started (and owns its shared memory) before anyone is sent
    // anything: arrive now, wait just before the first store to a peer
    if (!partials && splits > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    const int p = positions[seq];                 // one row per request: row index == request index
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int* bt = block_tables + (size_t)seq * max_pages;
    const int hi = p + 1;
    const int lo_key = first_key(p, window, SHAPED ? shape.chunk : 0);
    const int t_first = lo_key / BN;
    const int keep = KV1 ? shape.keep : 0;
    const int kt = KV1 ? min((keep + BN - 1) / BN, t_first) : 0;      // tiles of kept first tokens in front of the window's
    const int n_tiles = p >= 0 ? (hi + BN - 1) / BN - t_first + kt : 0;
    // the request's tile number n (0 .. n_tiles - 1) holds the keys from BN * tile_of(n) on
    auto tile_of = [&](int n) { return KV1 && n < kt ? n : t_first + n - kt; };
    if (partials) {
        splits = max(1, min(splits, n_tiles / DEC_MIN_TILES));
        const int share = max(1, (n_tiles + splits - 1) / splits);
        splits = max(1, (n_tiles + share - 1) / share);      // no block without a tile
        if (split >= splits) return;                  // the whole block: this request has no tiles for it
    }
    const int per = (n_tiles + splits - 1) / splits;
    const int n_begin = split * per;
    const int n_end = min(n_tiles, n_begin + per);
    // this block's pages: those of its tiles, BN / page_size of them each, one coalesced read of the block table
    const int ppt_shift = 6 - page_shift;
    for (int i = threadIdx.x; i < (max(n_end - n_begin, 0) << ppt_shift); i += NTHREADS) {
        const int lp = (tile_of(n_begin + (i >> ppt_shift)) << ppt_shift) + (i & ((1 << ppt_shift) - 1));
        s_pages[i] = lp <= (hi - 1) >> page_shift ? bt[lp] : 0;
    }
    __syncthreads();
    auto load_tile = [&](int n, int buf) {
        const int t = tile_of(n);
        const int* pages = s_pages + ((n - n_begin) << ppt_shift);
        load_kv_tile<HD, !KV1>(sK0 + buf * BN * LD, sV0 + buf * BN * LD, kc, vc, pages, t << ppt_shift, kvh, KV, page_shift, t * BN, lo_key, hi, keep);
        if (KV1) load_key_scales(sR0 + buf * BN, shape.kscale, pages, t << ppt_shift, page_shift, t * BN, lo_key, hi, keep);
    };

    // prologue: the first DEC_STAGES - 1 tiles, one commit group each (empty groups keep the
    // count); tiles that end before the newest key go out before the wait, the rest after it
    int s_done = 0;
#pragma unroll
    for (int s = 0; s < DEC_STAGES - 1; ++s) {
        int n = n_begin + s;
        if (s_done == s && (n >= n_end || (tile_of(n) + 1) * BN <= p)) {
            if (n < n_end) load_tile(n, s);
            cp_async_commit();
            s_done = s + 1;
        }
    }
    pdl_wait(8);
    // q of this step: plain loads (it must be in shared memory before the first tile is used, and
    // it is too small to deserve a commit group of its own)
    for (int c = threadIdx.x; c < 16 * (HD / 8); c += NTHREADS) {
        int r = c / (HD / 8), ch = c - r * (HD / 8);
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < G && p >= 0) v = *reinterpret_cast<const uint4*>(q + (size_t)seq * q_stride + (size_t)(kvh * G + r) * HD + ch * 8);
        *reinterpret_cast<uint4*>(sQ + r * LD + ch * 8) = v;
    }
#pragma unroll
    for (int s = 0; s < DEC_STAGES - 1; ++s) {
        if (s >= s_done) {
            int n = n_begin + s;
            if (n < n_end) load_tile(n, s);
            cp_async_commit();
        }
    }

    int pos[2], lo[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        int r = (lane >> 2) + h * 8;
        pos[h] = r < G ? p : -1;
        lo[h] = lo_key;
    }
    RowShape rs;
    if (SHAPED) {
        const int r0 = lane >> 2;
        rs = row_shape(shape, r0 < G ? kvh * G + r0 : -1, r0 + 8 < G ? kvh * G + r0 + 8 : -1);
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    float o[HD / 8][4];
#pragma unroll
    for (int n = 0; n < HD / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.f;
    uint32_t qf[HD / 16][4];

    for (int n = n_begin; n < n_end; ++n) {
        const int t = tile_of(n);
        int buf = (n - n_begin) % DEC_STAGES;
        __nv_bfloat16* sK = sK0 + buf * BN * LD;
        __nv_bfloat16* sV = sV0 + buf * BN * LD;
        cp_async_wait<DEC_STAGES - 2>();        // tile n has landed (one newer group may be in flight)
        __syncthreads();                        // ... for every thread; and everyone is done with tile n-1
        {
            int nn = n + DEC_STAGES - 1;        // refill the buffer tile n-1 used
            if (nn < n_end) load_tile(nn, (nn - n_begin) % DEC_STAGES);
            cp_async_commit();
        }
        if (n == n_begin) {
#pragma unroll
            for (int kk = 0; kk < HD / 16; ++kk)
                ldmatrix_x4(qf[kk], sQ + ((lane & 7) + ((lane >> 3) & 1) * 8) * LD + kk * 16 + (lane >> 4) * 8);
        }
        float s[2][4];
        qk_tile<HD, 2>(s, qf, sK, warp * 2);                    // this warp's 16 keys of the tile
        uint32_t pa[1][4];
        softmax_step<2, HD / 8, true, SHAPED, KV1>(s, pa, o, m, l, t * BN + warp * 16, lo, pos, scale_log2, &shape, &rs,
                                                   sR0 + buf * BN + warp * 16);
        pv_tile<HD, 1>(o, pa, sV, warp);
    }
    cp_async_wait<0>();
    __syncthreads();                                            // K/V buffers are free: reuse them for the combine
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    }
    float* cm = reinterpret_cast<float*>(sK0);                  // [4 warps][16 rows] max
    float* cl = cm + 64;                                        // [4][16] sum
    float* co = cl + 64;                                        // [4][16][HD]
    float* fin = co + 4 * 16 * HD;                              // this block's partial: [16][HD] values, [16] max, [16] sum
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        int r = (lane >> 2) + h * 8;
        if ((lane & 3) == 0) { cm[warp * 16 + r] = m[h]; cl[warp * 16 + r] = l[h]; }
#pragma unroll
        for (int n = 0; n < HD / 8; ++n) {
            co[(warp * 16 + r) * HD + n * 8 + (lane & 3) * 2] = o[n][2 * h];
            co[(warp * 16 + r) * HD + n * 8 + (lane & 3) * 2 + 1] = o[n][2 * h + 1];
        }
    }
    __syncthreads();
    const bool push = splits > 1 && !partials;
    const int chunk = (G * HD + splits - 1) / splits;          // outputs each block of a cluster finishes
    if (push) asm volatile("barrier.cluster.wait.aligned;" ::: "memory");       // the peers have started (they arrived at their start)
    for (int e = threadIdx.x; e < G * HD; e += NTHREADS) {
        int r = e / HD, d = e - r * HD;
        float M = fmaxf(fmaxf(cm[r], cm[16 + r]), fmaxf(cm[32 + r], cm[48 + r]));
        float Ms = M == -INFINITY ? 0.f : M;
        float acc = 0.f, L = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            float f = exp2f(cm[w * 16 + r] - Ms);
            acc += f * co[(w * 16 + r) * HD + d];
            L += f * cl[w * 16 + r];
        }
        if (splits == 1) {
            L = tail_den(tail, kvh * G + r, L, Ms);
            out[(size_t)seq * out_stride + (size_t)(kvh * G + r) * HD + d] =
                __float2bfloat16_rn(L > 0.f ? tail_val(tail, seq, kvh * G + r, (kvh * G + r) * HD + d, acc / L) : 0.f);
        } else if (push) {
            // to the block that finishes this output; the row's maximum and sum to every block
            const int owner = e / chunk;
            uint32_t dst;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"(smem_u32(recv_val + split * chunk + (e - owner * chunk))), "r"(owner));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(acc) : "memory");
            if (d == 0) {
                for (int k = 0; k < splits; ++k) {
                    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"(smem_u32(recv_m + split * 16 + r)), "r"(k));
                    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(M) : "memory");
                    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst + 128 * 4), "f"(L) : "memory");
                }
            }
        } else {
            fin[r * HD + d] = acc;
            if (d == 0) { fin[16 * HD + r] = M; fin[16 * HD + 16 + r] = L; }
        }
    }
    if (splits > 1 && partials) {
        float* mine = partials + ((size_t)(seq * KV + kvh) * gridDim.z + split) * PART;
        __syncthreads();
        for (int e = threadIdx.x; e < G * HD; e += NTHREADS) mine[e] = fin[e];
        if (threadIdx.x < 32) mine[16 * HD + threadIdx.x] = fin[16 * HD + threadIdx.x];
        __threadfence();
        __syncthreads();
        if (threadIdx.x == 0) s_last = atomicAdd(arrived + seq * KV + kvh, 1) == splits - 1;
        __syncthreads();
        if (!s_last) return;
        __threadfence();
        merge_partials<HD>(partials + (size_t)(seq * KV + kvh) * gridDim.z * PART, splits, G, reinterpret_cast<float*>(sK0),
                           out + (size_t)seq * out_stride + (size_t)kvh * G * HD, tail, seq, kvh * G);
        if (threadIdx.x == 0) arrived[seq * KV + kvh] = 0;      // ready for the next launch
    } else if (splits > 1) {
        // what was sent is there once everyone has passed this barrier
        asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
        const int total = G * HD;
        const int e0 = split * chunk, e1 = min(total, e0 + chunk);
        for (int e = e0 + threadIdx.x; e < e1; e += NTHREADS) {
            int r = e / HD, d = e - r * HD;
            float pm[8], pl[8], po[8];
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                pm[k] = -INFINITY; pl[k] = 0.f; po[k] = 0.f;
                if (k < splits) { po[k] = recv_val[k * chunk + (e - e0)]; pm[k] = recv_m[k * 16 + r]; pl[k] = recv_l[k * 16 + r]; }
            }
            float M = -INFINITY;
#pragma unroll
            for (int k = 0; k < 8; ++k) M = fmaxf(M, pm[k]);
            float Ms = M == -INFINITY ? 0.f : M;
            float acc = 0.f, L = 0.f;
#pragma unroll
            for (int k = 0; k < 8; ++k) {                       // rank order; ranks beyond the last add zero
                float f = exp2f(pm[k] - Ms);
                acc += f * po[k];
                L += f * pl[k];
            }
            L = tail_den(tail, kvh * G + r, L, Ms);
            out[(size_t)seq * out_stride + (size_t)(kvh * G + r) * HD + d] =
                __float2bfloat16_rn(L > 0.f ? tail_val(tail, seq, kvh * G + r, (kvh * G + r) * HD + d, acc / L) : 0.f);
        }
        // nothing of this block is read by a peer: it may leave at once
    }
}

template <int HD> constexpr size_t prefill_smem() { return (size_t)(64 + 4 * BN) * (HD + 8) * sizeof(__nv_bfloat16); }
template <int HD, int DEC_STAGES, bool KV1> size_t decode_smem(int G, bool cluster) {
    return decode_ring_bytes<HD, DEC_STAGES, KV1>() + (cluster ? decode_recv_bytes(G, HD) : 0);
}

inline int log2_exact(int v) {
    int s = 0;
    while ((1 << s) < v) ++s;
    return s;
}

// Raise a kernel's dynamic shared-memory limit when a launch needs more than any before it.
template <typename Kern>
int ensure_smem(Kern kernel, size_t bytes, size_t* configured) {
    if (bytes > 227 * 1024) return VOB_ERR_UNSUPPORTED;
    if (bytes > *configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
        if (e != cudaSuccess) return (int)e;
        *configured = bytes;
    }
    return 0;
}

template <int HD>
int launch_prefill(const void* q, long long q_stride, void* out, long long out_stride, const void* kc, const void* vc,
                   const int* bt, int max_pages, const int* seq_starts, const int* context_lens, int S, int max_new,
                   int H, int KV, int page_size, int window, float scale, AttnTail tail, cudaStream_t stream) {
    static size_t configured = 0;
    size_t smem = prefill_smem<HD>() + (size_t)max_pages * sizeof(int);      // tiles + this request's page list
    int e = ensure_smem(attn_prefill_mma_kernel<HD>, smem, &configured);
    if (e) return e;
    int G = H / KV;
    const long long row_tiles = ((long long)max_new * G + 63) / 64;
    if (row_tiles > 65535) return VOB_ERR_UNSUPPORTED;
    dim3 grid(KV, S, (unsigned)row_tiles);
    return vob_launch(attn_prefill_mma_kernel<HD>, grid, dim3(NTHREADS), smem, stream,
        (const __nv_bfloat16*)q, q_stride, (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)kc,
        (const __nv_bfloat16*)vc, bt, max_pages, seq_starts, context_lens, H, KV, log2_exact(page_size), window,
        scale * 1.4426950408889634f, tail);
}

template <int HD, int ST, bool SHAPED, bool KV1>
int launch_decode_st(const void* q, long long q_stride, void* out, long long out_stride, const void* kc, const void* vc,
                     const int* bt, int max_pages, const int* positions, int S, int H, int KV, int page_size, int window,
                     float scale, int splits, float* partials, int* arrived, AttnTail tail, ScoreShape shape, cudaStream_t stream) {
    static size_t configured = 0;
    // a block's page list: its share of the tiles of the longest request the block table can hold
    // (a request with few tiles uses fewer blocks, but then the tiles are few)
    long long tiles_max = ((long long)max_pages * page_size + BN - 1) / BN;
    long long per_max = (tiles_max + splits - 1) / splits;
    if (partials && per_max < 2 * DEC_MIN_TILES) per_max = 2 * DEC_MIN_TILES;
    long long pages_cta = per_max * (BN / page_size) + 1;
    size_t smem = decode_smem<HD, ST, KV1>(H / KV, splits > 1 && !partials) + (size_t)pages_cta * sizeof(int);
    int e = ensure_smem(attn_decode_mma_kernel<HD, ST, SHAPED, KV1>, smem, &configured);
    if (e) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(S, KV, splits);
    cfg.blockDim = dim3(NTHREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = partials ? 1 : splits;      // the blocks that share one (request, kv head)
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = g_vob_pdl ? 2 : 1;
    cudaError_t ce = cudaLaunchKernelEx(&cfg, attn_decode_mma_kernel<HD, ST, SHAPED, KV1>, (const __nv_bfloat16*)q, q_stride, (__nv_bfloat16*)out,
                                        out_stride, (const __nv_bfloat16*)kc, (const __nv_bfloat16*)vc, bt, max_pages, positions,
                                        H, KV, log2_exact(page_size), window, scale * 1.4426950408889634f, partials, arrived, tail, shape);
    return ce != cudaSuccess ? (int)ce : vob_launch_status();
}

template <int HD, bool SHAPED, bool KV1 = false>
int launch_decode(const void* q, long long q_stride, void* out, long long out_stride, const void* kc, const void* vc,
                  const int* bt, int max_pages, const int* positions, int S, int H, int KV, int page_size, int window,
                  float scale, int splits, float* partials, int* arrived, AttnTail tail, ScoreShape shape, cudaStream_t stream) {
    static int num_sms = 0;
    if (!num_sms) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, dev);
        if (num_sms <= 0) num_sms = 148;
    }
    // three stages while every block of the grid can be resident at once with them; else two
    long long blocks = (long long)S * KV * splits;
    long long fit3 = (long long)num_sms * ((227 * 1024) / (long long)(decode_smem<HD, 3, KV1>(H / KV, splits > 1 && !partials) + 2048));
    if (blocks <= fit3)
        return launch_decode_st<HD, 3, SHAPED, KV1>(q, q_stride, out, out_stride, kc, vc, bt, max_pages, positions, S, H, KV, page_size,
                                               window, scale, splits, partials, arrived, tail, shape, stream);
    return launch_decode_st<HD, 2, SHAPED, KV1>(q, q_stride, out, out_stride, kc, vc, bt, max_pages, positions, S, H, KV, page_size,
                                           window, scale, splits, partials, arrived, tail, shape, stream);
}

template <int HD, int HDV, bool SHAPED, bool KV1>
int launch_prefill_any(const void* q, long long q_stride, void* out, long long out_stride, const void* kc, const void* vc,
                       const int* bt, int max_pages, const int* seq_starts, const int* context_lens, int S, int max_new,
                       int H, int KV, int D, int DV, int page_size, int window, float scale, AttnTail tail, ScoreShape shape,
                       cudaStream_t stream) {
    static size_t configured = 0;
    size_t smem = ((size_t)(64 + 2 * BN) * (HD + 8) + (KV1 ? (size_t)0 : (size_t)2 * BN * (HDV + 8))) * sizeof(__nv_bfloat16) +
                  (KV1 ? 2 * BN * sizeof(float) : 0) + (size_t)2 * max_pages * sizeof(int);
    int e = ensure_smem(attn_prefill_mma_any_kernel<HD, HDV, SHAPED, KV1>, smem, &configured);
    if (e) return e;
    const long long row_tiles = ((long long)max_new * (H / KV) + 63) / 64;
    if (row_tiles > 65535) return VOB_ERR_UNSUPPORTED;
    dim3 grid(KV, S, (unsigned)row_tiles);
    return vob_launch(attn_prefill_mma_any_kernel<HD, HDV, SHAPED, KV1>, grid, dim3(NTHREADS), smem, stream,
        (const __nv_bfloat16*)q, q_stride, (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)kc,
        (const __nv_bfloat16*)vc, bt, max_pages, seq_starts, context_lens, H, KV, D, DV, log2_exact(page_size), window,
        scale * 1.4426950408889634f, tail, shape);
}

bool sizes_ok(int H, int KV, int hd, int page_size) {
    return (hd == 64 || hd == 128) && KV > 0 && H % KV == 0 && page_size > 0 && BN % page_size == 0;
}

// The checks and the choice of tile widths of the portion kernel for keys and values of sizes of their own.
template <bool SHAPED>
int prefill_any(const void* q, long long q_stride, void* out, long long out_stride, const void* kcache, const void* vcache,
                const int* block_tables, int max_pages, const int* seq_starts, const int* context_lens, int S, int max_new, int H,
                int KV, int D, int DV, int page_size, int window, float scale, AttnTail tail, ScoreShape shape, cudaStream_t stream) {
    if (S <= 0 || max_new <= 0) return 0;
    if (KV <= 0 || H % KV != 0 || page_size <= 0 || BN % page_size != 0) return VOB_ERR_UNSUPPORTED;
    if (D <= 0 || DV <= 0 || D % 8 != 0 || DV % 8 != 0 || D > 128 || DV > 128) return VOB_ERR_UNSUPPORTED;
    if (q_stride % 8 != 0 || out_stride % 2 != 0 || S > 65535 || KV > 65535) return VOB_ERR_BAD_ARG;
    if (SHAPED && kcache == vcache) {          // the values are the cached keys
        if (D != DV || shape.pool > 0) return VOB_ERR_BAD_ARG;
#define VOB_KV1(HD_)                                                                                                                \
    return launch_prefill_any<HD_, HD_, true, true>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages,           \
                                                    seq_starts, context_lens, S, max_new, H, KV, D, DV, page_size, window, scale,    \
                                                    tail, shape, stream)
        if (D <= 32) VOB_KV1(32);
        if (D <= 64) VOB_KV1(64);
        if (D <= 96) VOB_KV1(96);
        VOB_KV1(128);
#undef VOB_KV1
    }
#define VOB_ANY(HD_, HDV_)                                                                                                          \
    return launch_prefill_any<HD_, HDV_, SHAPED, false>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, seq_starts,  \
                                                 context_lens, S, max_new, H, KV, D, DV, page_size, window, scale, tail, shape, stream)
#define VOB_ANY_V(HD_)                                                                                                              \
    do {                                                                                                                            \
        if (DV <= 32) VOB_ANY(HD_, 32);                                                                                             \
        if (DV <= 64) VOB_ANY(HD_, 64);                                                                                             \
        VOB_ANY(HD_, 128);                                                                                                          \
    } while (0)
    if (D <= 32) VOB_ANY_V(32);
    if (D <= 64) VOB_ANY_V(64);
    if (D <= 96) VOB_ANY_V(96);
    VOB_ANY_V(128);
#undef VOB_ANY_V
#undef VOB_ANY
}

}  // namespace

// 1 if the tensor-core kernels take these sizes (decode additionally needs H / KV <= 16).
VOB_EXPORT int vob_attn_mma_supported(int H, int KV, int hd, int page_size, int decode) {
    if (!sizes_ok(H, KV, hd, page_size)) return 0;
    if (decode && H / KV > 16) return 0;
    return 1;
}

VOB_EXPORT int vob_attn_prefill_mma(const void* q, long long q_stride, void* out, long long out_stride, const void* kcache,
                                    const void* vcache, const int* block_tables, int max_pages, const int* seq_starts,
                                    const int* context_lens, int S, int max_new, int H, int KV, int hd, int page_size,
                                    int window, float scale, const float* sink, const void* gate, long long gate_stride,
                                    float out_scale, cudaStream_t stream) {
    const AttnTail tail{sink, (const __nv_bfloat16*)gate, gate_stride, out_scale, 0};
    if (S <= 0 || max_new <= 0) return 0;
    if (!sizes_ok(H, KV, hd, page_size)) return VOB_ERR_UNSUPPORTED;
    if (q_stride % 8 != 0 || out_stride % 2 != 0 || S > 65535 || KV > 65535) return VOB_ERR_BAD_ARG;
    if (hd == 64) return launch_prefill<64>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, seq_starts,
                                           context_lens, S, max_new, H, KV, page_size, window, scale, tail, stream);
    return launch_prefill<128>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, seq_starts,
                               context_lens, S, max_new, H, KV, page_size, window, scale, tail, stream);
}

// Portions of prompts and mixed batches with keys of D and values of DV features, multiples of 8 up to 128 each
// (kcache [pages, KV, page_size, D], vcache [pages, KV, page_size, DV]); everything else as vob_attn_prefill_mma.
VOB_EXPORT int vob_attn_prefill_mma_any(const void* q, long long q_stride, void* out, long long out_stride, const void* kcache,
                                        const void* vcache, const int* block_tables, int max_pages, const int* seq_starts,
                                        const int* context_lens, int S, int max_new, int H, int KV, int D, int DV, int page_size,
                                        int window, float scale, const float* sink, const void* gate, long long gate_stride,
                                        float out_scale, cudaStream_t stream) {
    const AttnTail tail{sink, (const __nv_bfloat16*)gate, gate_stride, out_scale, 0};
    return prefill_any<false>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, seq_starts, context_lens, S, max_new,
                              H, KV, D, DV, page_size, window, scale, tail, make_shape(0, 0.f, nullptr, nullptr, scale), stream);
}

// The checked arguments of the shaped forms. r1 without r2: a linear bias. `keep` goes with a window; `kscale` with values
// that are the cached keys (kcache == vcache).
static int shape_args_ok(int chunk, float softcap, const float* r1, const float* r2, int keep, int window, const float* kscale,
                         const void* kcache, const void* vcache) {
    if (chunk < 0 || softcap < 0.f || (r2 && !r1)) return 0;
    if (keep < 0 || (keep > 0 && (window <= 0 || chunk > 0))) return 0;
    // the kernels whose values are the cached keys take a linear bias, kept first tokens and a number per key; the others none of them
    if (kcache != vcache) return !(kscale || keep > 0 || (r1 && !r2));
    return !r2;
}

// The same with scores that are shaped before the softmax: a query reads the keys of its own block of `chunk` positions
// (0: no blocks), score <- softcap * tanh(score / softcap) (0: no cap), r1[head] * ln(1 + r2[head] * distance) is taken
// off (r1, r2 float32 [H], or both null). Any sign of `scale`. kcache == vcache: the values are the cached keys; then r1[head] *
// distance is taken off (r2 null), q . k is multiplied by kscale [pages][page_size] (null: by nothing), and the first `keep` keys are
// seen whatever the window. `gate_heads`: the gate has one column per head.
VOB_EXPORT int vob_attn_prefill_shaped(const void* q, long long q_stride, void* out, long long out_stride, const void* kcache,
                                       const void* vcache, const int* block_tables, int max_pages, const int* seq_starts,
                                       const int* context_lens, int S, int max_new, int H, int KV, int D, int DV, int page_size,
                                       int window, float scale, const float* sink, const void* gate, long long gate_stride,
                                       float out_scale, int chunk, float softcap, const float* r1, const float* r2,
                                       const void* kpool, const void* vpool, int pool, int keep, const float* kscale, int gate_heads,
                                       cudaStream_t stream) {
    const AttnTail tail{sink, (const __nv_bfloat16*)gate, gate_stride, out_scale, gate_heads};
    if (!shape_args_ok(chunk, softcap, r1, r2, keep, window, kscale, kcache, vcache)) return VOB_ERR_BAD_ARG;
    // pooled entries (kpool, vpool laid out like the caches, `pool` tokens an entry) go with a window, without blocks of
    // positions and without a distance bias
    if (pool < 0 || (pool > 0) != (kpool != nullptr) || (kpool != nullptr) != (vpool != nullptr)) return VOB_ERR_BAD_ARG;
    if (pool > 0 && (window <= 0 || chunk > 0 || r1 || keep > 0)) return VOB_ERR_BAD_ARG;
    const ScoreShape shape = make_shape(chunk, softcap, r1, r2, scale, kpool, vpool, pool, keep, r1 && !r2, kscale);
    return prefill_any<true>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, seq_starts, context_lens, S, max_new,
                             H, KV, D, DV, page_size, window, scale, tail, shape, stream);
}

// `splits` (1..8) blocks share each (request, kv head) as one cluster. With `partials` (float32
// [S * KV * splits * (16 * hd + 32)]) and `arrived` (int32 [S * KV], zero; left zero) up to 64 blocks
// share it without a cluster and merge through global memory.
VOB_EXPORT int vob_attn_decode_mma(const void* q, long long q_stride, void* out, long long out_stride, const void* kcache,
                                   const void* vcache, const int* block_tables, int max_pages, const int* positions, int S,
                                   int H, int KV, int hd, int page_size, int window, float scale, int splits,
                                   void* partials, int* arrived, const float* sink, const void* gate, long long gate_stride,
                                   float out_scale, cudaStream_t stream) {
    const AttnTail tail{sink, (const __nv_bfloat16*)gate, gate_stride, out_scale, 0};
    const ScoreShape none = make_shape(0, 0.f, nullptr, nullptr, scale);
    if (S <= 0) return 0;
    if (!sizes_ok(H, KV, hd, page_size) || H / KV > 16) return VOB_ERR_UNSUPPORTED;
    if ((partials == nullptr) != (arrived == nullptr)) return VOB_ERR_BAD_ARG;
    if (q_stride % 8 != 0 || splits < 1 || splits > (partials ? DEC_MAX_SPLITS_WIDE : 8) || KV > 65535) return VOB_ERR_BAD_ARG;
    if (hd == 64) return launch_decode<64, false>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, positions, S,
                                                 H, KV, page_size, window, scale, splits, (float*)partials, arrived, tail, none, stream);
    return launch_decode<128, false>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, positions, S, H, KV,
                                     page_size, window, scale, splits, (float*)partials, arrived, tail, none, stream);
}

// vob_attn_decode_mma with shaped scores (see vob_attn_prefill_shaped).
VOB_EXPORT int vob_attn_decode_shaped(const void* q, long long q_stride, void* out, long long out_stride, const void* kcache,
                                      const void* vcache, const int* block_tables, int max_pages, const int* positions, int S,
                                      int H, int KV, int hd, int page_size, int window, float scale, int splits,
                                      void* partials, int* arrived, const float* sink, const void* gate, long long gate_stride,
                                      float out_scale, int chunk, float softcap, const float* r1, const float* r2,
                                      int keep, const float* kscale, int gate_heads, cudaStream_t stream) {
    const AttnTail tail{sink, (const __nv_bfloat16*)gate, gate_stride, out_scale, gate_heads};
    if (S <= 0) return 0;
    if (!shape_args_ok(chunk, softcap, r1, r2, keep, window, kscale, kcache, vcache)) return VOB_ERR_BAD_ARG;
    const ScoreShape shape = make_shape(chunk, softcap, r1, r2, scale, nullptr, nullptr, 0, keep, r1 && !r2, kscale);
    if (!sizes_ok(H, KV, hd, page_size) || H / KV > 16) return VOB_ERR_UNSUPPORTED;
    if ((partials == nullptr) != (arrived == nullptr)) return VOB_ERR_BAD_ARG;
    if (q_stride % 8 != 0 || splits < 1 || splits > (partials ? DEC_MAX_SPLITS_WIDE : 8) || KV > 65535) return VOB_ERR_BAD_ARG;
    if (kcache == vcache) {                    // the values are the cached keys
        if (hd == 64) return launch_decode<64, true, true>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, positions, S,
                                                          H, KV, page_size, window, scale, splits, (float*)partials, arrived, tail, shape, stream);
        return launch_decode<128, true, true>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, positions, S, H, KV,
                                              page_size, window, scale, splits, (float*)partials, arrived, tail, shape, stream);
    }
    if (hd == 64) return launch_decode<64, true>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, positions, S,
                                                H, KV, page_size, window, scale, splits, (float*)partials, arrived, tail, shape, stream);
    return launch_decode<128, true>(q, q_stride, out, out_stride, kcache, vcache, block_tables, max_pages, positions, S, H, KV,
                                    page_size, window, scale, splits, (float*)partials, arrived, tail, shape, stream);
}
