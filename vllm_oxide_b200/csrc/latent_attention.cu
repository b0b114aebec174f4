// Attention over a latent cache: per token the pages hold ONE latent vector c (width L, shared by
// all heads, already normalised) and ONE rotated key part (width R, shared by all heads), not
// keys and values per head. A head's key is [W_uk c | rotated part] and its value W_uv c, but
// neither is ever built: with q_lat = W_uk^T q_plain (done by the caller as a matrix product)
//     score(i, j) = (q_lat_i . c_j + q_rot_i . kr_j) * scale,   out_lat_i = sum_j softmax_j(score) c_j
// and the caller applies W_uv to out_lat. Causal: row i of a request sees the keys 0 .. position(i)
// of that request, all read from the pages (the step's own tokens were written first).
//
// vob_latent_prep: per token, any of three jobs: c = weight * x / sqrt(mean(x^2) + eps) of the first L
// columns of the down projection and the rotary positions on its last R columns, both written to the
// token's cache slot; the rotated query part of every head to a float32 buffer; the same norm on a
// latent the queries are made from (designs whose queries go through one), to a buffer of its own.
// vob_latent_gate: the heads' values times sigmoid(gate), element by element, put side by side per token.
// vob_latent_attend: scores, softmax weights and the weighted sum in float32, keys in page order
// from the first, in tiles staged in shared memory; one warp per head, a block takes up to 8 heads
// of one row, so a key tile is read once for all of them. The order of every sum depends only on the row's
// position, never on how the request was cut into steps or on the batch around it. Steps of few rows
// (single tokens) share a row's keys over `splits` blocks, whose partial results a second small kernel
// puts together in a fixed order.
#include "common.cuh"
#include <math.h>
VOB_PDL_SWITCH(latent_attention)

// q [T, ld_q]: the query of head h at columns h * (D + R) (D plain features, then R to be rotated); down [T, ld]: the down
// projection's L + R columns. lat [pages, 1, page, L], kr [pages, 1, page, R] in the cache's type TC. q_rot float32 [T, H, R].
// Cosine and sine are both multiplied by `mag`. Rows with position < 0 write nothing (their q_rot is zero); a slot < 0 writes
// no cache. `q` null: no queries here; `slots` null: no cache write; `low` [T, ld_low] (Q columns) null: no query latent, else
// low_out [T, Q] = low_w * low / sqrt(mean(low^2) + eps), every row.
// Launch: grid (tokens, blocks that share a token's queries), 128 threads; the first block of a token does the rest.
template <typename T, typename TC>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const T* __restrict__ q, long ld_q, int H, int D, int R, const T* __restrict__ down_p, long ld, int L,
                   const float* __restrict__ norm_w, float eps, const int* __restrict__ positions, const int* __restrict__ slots,
                   const float* __restrict__ inv_freq, float mag, TC* __restrict__ lat, TC* __restrict__ kr, float* __restrict__ q_rot,
                   const T* __restrict__ low, long ld_low, int Q, const float* __restrict__ low_w, T* __restrict__ low_out) {
    pdl_launch_dependents();
    pdl_wait(45);
    __shared__ float red[4], red_low[4];
    const int t = blockIdx.x, tid = threadIdx.x;
    const int pos = positions[t];
    const int half = R >> 1;
    if (q) {
        const T* row = q + (size_t)t * ld_q;
        float* qo = q_rot + (size_t)t * H * R;
        // a thread takes a pair of features: its angle's cosine and sine serve both
        for (int e = blockIdx.y * blockDim.x + tid; e < H * half; e += blockDim.x * gridDim.y) {
            const int h = e / half, i = e - h * half;
            float u = 0.f, v = 0.f;
            if (pos >= 0) {
                const float ang = (float)pos * inv_freq[i];
                const float cs = cosf(ang) * mag, sn = sinf(ang) * mag;
                const T* qh = row + (size_t)h * (D + R) + D;
                const float a = ld_f(qh + i), b = ld_f(qh + i + half);
                u = a * cs - b * sn;
                v = b * cs + a * sn;
            }
            qo[h * R + i] = u;
            qo[h * R + i + half] = v;
        }
    }
    if (blockIdx.y > 0) return;
    const int slot = slots ? slots[t] : -1;
    const bool write = pos >= 0 && slot >= 0;
    if (!write && !low) return;
    const T* down = down_p + (size_t)t * ld;
    const T* lrow = low + (size_t)t * ld_low;
    float ss = 0.f, sl = 0.f;
    if (write)
        for (int i = tid; i < L; i += blockDim.x) {
            const float x = ld_f(down + i);
            ss = fmaf(x, x, ss);
        }
    if (low)
        for (int i = tid; i < Q; i += blockDim.x) {
            const float x = ld_f(lrow + i);
            sl = fmaf(x, x, sl);
        }
    ss = warp_sum(ss);
    sl = warp_sum(sl);
    if ((tid & 31) == 0) { red[tid >> 5] = ss; red_low[tid >> 5] = sl; }
    __syncthreads();
    if (low) {
        const float inv = 1.0f / sqrtf(((red_low[0] + red_low[1]) + (red_low[2] + red_low[3])) / (float)Q + eps);
        T* o = low_out + (size_t)t * Q;
        for (int i = tid; i < Q; i += blockDim.x) st_f(o + i, low_w[i] * (ld_f(lrow + i) * inv));
    }
    if (!write) return;
    const float inv = 1.0f / sqrtf(((red[0] + red[1]) + (red[2] + red[3])) / (float)L + eps);
    TC* lo = lat + (size_t)slot * L;
    for (int i = tid; i < L; i += blockDim.x) st_f(lo + i, norm_w[i] * (ld_f(down + i) * inv));
    TC* ko = kr + (size_t)slot * R;
    for (int f = tid; f < R; f += blockDim.x) {
        const int i = f < half ? f : f - half;
        const float ang = (float)pos * inv_freq[i];
        const float cs = cosf(ang) * mag, sn = sinf(ang) * mag;
        const float a = ld_f(down + L + i), b = ld_f(down + L + i + half);
        st_f(ko + f, f < half ? a * cs - b * sn : b * cs + a * sn);
    }
}

VOB_EXPORT int vob_latent_prep(const void* q, int code, long ld_q, int H, int D, int R, const void* down, long ld, int L,
                               const float* norm_w, float eps, const int* positions, const int* slots, const float* inv_freq, float mag,
                               void* lat, void* kr, int cache_code, float* q_rot, const void* low, long ld_low, int Q, const float* low_w,
                               void* low_out, int T, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || D < 0 || R <= 0 || (R & 1) || L <= 0 || code != cache_code) return VOB_ERR_BAD_ARG;
    if ((q && !q_rot) || (slots && (!down || !lat || !kr)) || (low && (Q <= 0 || !low_w || !low_out))) return VOB_ERR_BAD_ARG;
    const int pairs = H * (R / 2), by = !q ? 1 : pairs <= 128 ? 1 : pairs >= 1024 ? 8 : (pairs + 127) / 128;
    VOB_DISPATCH_ELEM(code, return vob_launch(latent_prep_kernel<ElemT, ElemT>, dim3(T, by), dim3(128), 0, stream, (const ElemT*)q, ld_q, H, D, R,
                                              (const ElemT*)down, ld, L, norm_w, eps, positions, slots, inv_freq, mag, (ElemT*)lat,
                                              (ElemT*)kr, q_rot, (const ElemT*)low, ld_low, Q, low_w, (ElemT*)low_out));
    return 0;
}

// ---------------------------------------------------------------------------------------------
// out[t, h * V + i] = vals(t, h, i) * sigmoid(gate[t, h * V + i]); vals at t * v_ts + h * v_hs + i, gate rows ld_gate apart, out
// [T, H * V] (may be vals itself where that has its layout). PER elements (16 bytes) a thread where sizes and addresses allow.
// Launch: grid (rows, ceil(H V / (256 PER))). Bound: memory.
// ---------------------------------------------------------------------------------------------
template <typename T, int PER>
__global__ void __launch_bounds__(256)
latent_gate_kernel(const T* vals, long v_ts, long v_hs, const T* __restrict__ gate, long ld_gate, int H, int V, T* out) {
    pdl_launch_dependents();
    pdl_wait(49);
    const int t = blockIdx.x, e = (blockIdx.y * 256 + threadIdx.x) * PER;
    if (e >= H * V) return;
    const int h = e / V, i = e - h * V;
    const T* src = vals + (size_t)t * v_ts + (size_t)h * v_hs + i;
    const T* g = gate + (size_t)t * ld_gate + e;
    T* o = out + (size_t)t * H * V + e;
    if constexpr (PER == 1) {
        st_f(o, ld_f(src) / (1.0f + expf(-ld_f(g))));
    } else {
        T a[PER], b[PER];
        *reinterpret_cast<uint4*>(a) = *reinterpret_cast<const uint4*>(src);
        *reinterpret_cast<uint4*>(b) = *reinterpret_cast<const uint4*>(g);
#pragma unroll
        for (int k = 0; k < PER; ++k) st_f(a + k, ld_f(a + k) / (1.0f + expf(-ld_f(b + k))));
        *reinterpret_cast<uint4*>(o) = *reinterpret_cast<const uint4*>(a);
    }
}

VOB_EXPORT int vob_latent_gate(const void* vals, int code, long v_ts, long v_hs, const void* gate, long ld_gate, int T, int H, int V,
                               void* out, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || V <= 0 || (H * V + 255) / 256 > 65535) return VOB_ERR_BAD_ARG;
    const int per = code == VOB_BF16 ? 8 : 4;
    if (V % per == 0 && v_ts % per == 0 && v_hs % per == 0 && ld_gate % per == 0 && (((uintptr_t)vals | (uintptr_t)gate | (uintptr_t)out) & 15) == 0) {
        const dim3 grid(T, (H * V / per + 255) / 256);
        if (code == VOB_BF16)
            return vob_launch(latent_gate_kernel<__nv_bfloat16, 8>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)vals, v_ts, v_hs,
                              (const __nv_bfloat16*)gate, ld_gate, H, V, (__nv_bfloat16*)out);
        if (code == VOB_F32)
            return vob_launch(latent_gate_kernel<float, 4>, grid, dim3(256), 0, stream, (const float*)vals, v_ts, v_hs, (const float*)gate,
                              ld_gate, H, V, (float*)out);
        return VOB_ERR_BAD_ARG;
    }
    VOB_DISPATCH_ELEM(code, return vob_launch(latent_gate_kernel<ElemT, 1>, dim3(T, (H * V + 255) / 256), dim3(256), 0, stream, (const ElemT*)vals, v_ts,
                                              v_hs, (const ElemT*)gate, ld_gate, H, V, (ElemT*)out));
    return 0;
}

// q_lat float32, element (t, h, i) at t * q_ts + h * q_hs + i; q_rot float32 [T, H, R]; out_lat of type
// TO, element (t, h, i) at t * o_ts + h * o_hs + i. NL = ceil(L / 32) registers per lane for q_lat and
// for the weighted sum. Grid (rows, ceil(H / warps)); a block has `warps` warps, one head each.
template <int NL, typename TC, typename TO>
__global__ void __launch_bounds__(256, 1)
latent_attend_kernel(const float* __restrict__ q_lat, long q_ts, long q_hs, const float* __restrict__ q_rot,
                     const TC* __restrict__ lat, const TC* __restrict__ kr, const int* __restrict__ block_tables, int max_pages,
                     const int* __restrict__ row_seq, const int* __restrict__ positions, int page_size, int H, int L, int R,
                     float scale, int KT, TO* __restrict__ out, long o_ts, long o_hs, int splits, float* __restrict__ part, int window) {
    pdl_launch_dependents();
    pdl_wait(46);
    extern __shared__ float tile[];                 // [KT][L + R]
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y * (blockDim.x >> 5) + warp;
    const bool head = h < H;
    const int pos = positions[t];
    TO* orow = out + (size_t)t * o_ts + (size_t)(head ? h : 0) * o_hs;
    // with splits > 1 block z takes the z-th share of the row's keys and leaves (max, sum, weighted sum) in `part`
    // [T, H, splits, L + 2]; the shares depend on the row's position and `splits` only
    float* prow = part + (((size_t)t * H + (head ? h : 0)) * splits + blockIdx.z) * (L + 2);
    if (pos < 0) {
        if (head && splits == 1)
            for (int i = lane; i < L; i += 32) st_f(orow + i, 0.f);
        if (head && splits > 1 && lane == 0) { prow[0] = -INFINITY; prow[1] = 0.f; }
        return;
    }
    const int* table = block_tables + (size_t)row_seq[t] * max_pages;
    const int W = L + R;
    float ql[NL], qr[4], acc[NL];
#pragma unroll
    for (int i = 0; i < NL; ++i) {
        const int c = lane + 32 * i;
        ql[i] = (head && c < L) ? q_lat[(size_t)t * q_ts + (size_t)h * q_hs + c] : 0.f;
        acc[i] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int c = lane + 32 * i;
        qr[i] = (head && c < R) ? q_rot[((size_t)t * H + h) * R + c] : 0.f;
    }
    float m = -INFINITY, l = 0.f;
    // the keys a row sees: all up to its own, or with a window only the last `window` of them
    const int first = window > 0 ? max(0, pos + 1 - window) : 0;
    const int share = ((pos - first + splits) / splits + KT - 1) / KT * KT;      // keys per block, whole tiles
    const int nkeys = min(pos + 1, first + (int)(blockIdx.z + 1) * share);
    for (int k0 = first + blockIdx.z * share; k0 < nkeys; k0 += KT) {
        const int n = min(KT, nkeys - k0);
        __syncthreads();
        // a warp copies whole keys (one page lookup per key, then consecutive elements)
        for (int kk = warp; kk < n; kk += (int)(blockDim.x >> 5)) {
            const int key = k0 + kk;
            const size_t slot = (size_t)table[key / page_size] * page_size + key % page_size;
            float* dst = tile + kk * W;
            for (int c = lane; c < L; c += 32) dst[c] = ld_f(lat + slot * L + c);
            for (int c = lane; c < R; c += 32) dst[L + c] = ld_f(kr + slot * R + c);
        }
        __syncthreads();
        // four keys at a time: their dot products and reductions are independent chains
        for (int kk = 0; kk < n; kk += 4) {
            float sc[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float* kv = tile + min(kk + j, n - 1) * W;
                float a = 0.f;
#pragma unroll
                for (int i = 0; i < NL; ++i) {
                    const int c = lane + 32 * i;
                    if (c < L) a = fmaf(ql[i], kv[c], a);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int c = lane + 32 * i;
                    if (c < R) a = fmaf(qr[i], kv[L + c], a);
                }
                sc[j] = a;
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
                for (int j = 0; j < 4; ++j) sc[j] += __shfl_xor_sync(0xffffffffu, sc[j], o);
            }
            float mn = m;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                sc[j] = kk + j < n ? sc[j] * scale : -INFINITY;
                mn = fmaxf(mn, sc[j]);
            }
            const float corr = expf(m - mn);            // exp(-inf) = 0 at the first keys
            float p[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) p[j] = expf(sc[j] - mn);
            l = fmaf(l, corr, (p[0] + p[1]) + (p[2] + p[3]));
#pragma unroll
            for (int i = 0; i < NL; ++i) {
                const int c = lane + 32 * i;
                float a = acc[i] * corr;
                if (c < L) {
#pragma unroll
                    for (int j = 0; j < 4; ++j) a = fmaf(p[j], tile[min(kk + j, n - 1) * W + c], a);
                }
                acc[i] = a;
            }
            m = mn;
        }
    }
    if (head && splits == 1) {
        const float inv = 1.0f / l;
#pragma unroll
        for (int i = 0; i < NL; ++i) {
            const int c = lane + 32 * i;
            if (c < L) st_f(orow + c, acc[i] * inv);
        }
    }
    if (head && splits > 1) {
        if (lane == 0) { prow[0] = m; prow[1] = l; }
#pragma unroll
        for (int i = 0; i < NL; ++i) {
            const int c = lane + 32 * i;
            if (c < L) prow[2 + c] = acc[i];
        }
    }
}

// The shares of a row's keys put together, in share order: out = sum_z acc_z e^(m_z - M) / sum_z l_z e^(m_z - M).
// Launch: one block of 128 threads per (row, head), at most VOB_LATENT_SPLITS shares.
#define VOB_LATENT_SPLITS 64
template <typename TO>
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part, const int* __restrict__ positions, int H, int L, int splits,
                    TO* __restrict__ out, long o_ts, long o_hs) {
    pdl_launch_dependents();
    pdl_wait(47);
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    TO* orow = out + (size_t)t * o_ts + (size_t)h * o_hs;
    const float* p = part + ((size_t)t * H + h) * splits * (L + 2);
    if (positions[t] < 0) {
        for (int i = tid; i < L; i += blockDim.x) st_f(orow + i, 0.f);
        return;
    }
    __shared__ float wgt[VOB_LATENT_SPLITS], total;
    if (tid < 32) {                    // one warp works out the shares' weights, two shares a lane
        float m[2], sum[2];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int z = tid + 32 * k;
            m[k] = z < splits ? p[(size_t)z * (L + 2)] : -INFINITY;
            sum[k] = z < splits ? p[(size_t)z * (L + 2) + 1] : 0.f;
        }
        const float M = warp_max(fmaxf(m[0], m[1]));
        float l = 0.f;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float w = sum[k] > 0.f ? expf(m[k] - M) : 0.f;            // 0: a share without keys, nothing of it is read
            if (tid + 32 * k < splits) wgt[tid + 32 * k] = w;
            l = fmaf(sum[k], w, l);
        }
        l = warp_sum(l);
        if (tid == 0) total = l;
    }
    __syncthreads();
    const float l = total;
    const float inv = 1.0f / l;
    for (int i = tid; i < L; i += blockDim.x) {
        float a = 0.f;
#pragma unroll 8
        for (int z = 0; z < splits; ++z) {
            const float v = wgt[z] > 0.f ? p[(size_t)z * (L + 2) + 2 + i] : 0.f;
            a = fmaf(v, wgt[z], a);
        }
        st_f(orow + i, a * inv);
    }
}

VOB_EXPORT int vob_latent_attend(const float* q_lat, long q_ts, long q_hs, const float* q_rot, const void* lat, const void* kr,
                                 int cache_code, const int* block_tables, int max_pages, const int* row_seq, const int* positions,
                                 int page_size, int T, int H, int L, int R, float scale, void* out, int out_code, long o_ts, long o_hs,
                                 int splits, float* part, int window, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (window < 0) return VOB_ERR_BAD_ARG;
    if (H <= 0 || L <= 0 || R <= 0 || page_size <= 0 || max_pages <= 0 || cache_code != out_code) return VOB_ERR_BAD_ARG;
    if (splits < 1 || splits > VOB_LATENT_SPLITS || (splits > 1 && !part) || H > 65535) return VOB_ERR_BAD_ARG;
    if (L > 1024 || R > 128) return VOB_ERR_UNSUPPORTED;
    const int warps = H < 8 ? H : 8;
    const int W = L + R;
    int KT = (int)(40 * 1024 / ((size_t)W * 4));
    KT = KT > 32 ? 32 : KT < 1 ? 1 : KT;
    const size_t smem = (size_t)KT * W * 4;
    dim3 grid(T, (H + warps - 1) / warps, splits), block(32 * warps);
    const int nl = (L + 31) / 32;
    int status = VOB_ERR_BAD_ARG;
#define VOB_LA(N, TC)                                                                                                          \
    status = vob_launch(latent_attend_kernel<N, TC, TC>, grid, block, smem, stream, q_lat, q_ts, q_hs, q_rot, (const TC*)lat, \
                        (const TC*)kr, block_tables, max_pages, row_seq, positions, page_size, H, L, R, scale, KT, (TC*)out, o_ts, o_hs, \
                        splits, part, window)
#define VOB_LA_N(TC)                       \
    do {                                   \
        if (nl <= 4) { VOB_LA(4, TC); }        \
        else if (nl <= 8) { VOB_LA(8, TC); }   \
        else if (nl <= 16) { VOB_LA(16, TC); } \
        else { VOB_LA(32, TC); }               \
        if (status == 0 && splits > 1)         \
            status = vob_launch(latent_merge_kernel<TC>, dim3(T, H), dim3(128), 0, stream, (const float*)part, positions, H, L, splits, \
                                (TC*)out, o_ts, o_hs);                                                                          \
    } while (0)
    if (cache_code == VOB_F32) VOB_LA_N(float);
    else if (cache_code == VOB_BF16) VOB_LA_N(__nv_bfloat16);
#undef VOB_LA_N
#undef VOB_LA
    return status;
}


// ---------------------------------------------------------------------------------------------
// Prompt portions in bfloat16 on the tensor cores (mma.sync m16n8k16, operands by ldmatrix). A block takes 16
// consecutive tokens of one request and HB heads; a head has WPH warps, each of which owns a share of the latent
// columns of O (at most 256) and computes the head's S = Q K^T for itself. A tile of 32 keys ([c | kr], L + R
// wide, bfloat16, rows padded by 16 bytes so that ldmatrix meets no bank conflict) is brought into shared memory
// once for all of them; the next tile is fetched into registers meanwhile. S, the softmax (float32, running
// maximum and sum per row), P (bfloat16, taken straight from S's registers as the next product's A operand) and
// O (float32) never leave the registers. Needs L and R multiples of 16. Rows are a request's seq_starts[s] + 16
// * tile ..; their positions are consecutive, so the tile's last row bounds the keys and every row masks what
// lies behind its own position.
//
// Steps of single tokens run the same kernel with HEADS: the 16 rows of a tile are 16 heads of ONE token (they share its
// keys), the warps of a block share out the latent columns, and `splits` blocks share a token's keys in whole tiles; with more
// than one share each leaves (max, sum, weighted sum) per head in `part` for latent_merge_kernel, as latent_attend_kernel does.
// ---------------------------------------------------------------------------------------------
#define VOB_LTC_BN 32
#define VOB_LTC_PRE 10        // 16-byte pieces of the next key tile a thread holds ahead (the rest of a tile is copied when it is due)

__device__ __forceinline__ void ldsm_x4(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void ldsm_x4_trans(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void mma_bf16_16816(float* c, unsigned a0, unsigned a1, unsigned a2, unsigned a3, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned*>(&v);
}

// NT16: groups of 16 latent columns a warp owns at most (its O accumulator is NT16 * 8 registers).
template <int NT16, bool HEADS>
__global__ void __launch_bounds__(256, HEADS && NT16 <= 4 ? 2 : 1)
latent_attend_tc_kernel(const float* __restrict__ q_lat, long q_ts, long q_hs, const float* __restrict__ q_rot,
                        const __nv_bfloat16* __restrict__ lat, const __nv_bfloat16* __restrict__ kr, const int* __restrict__ block_tables,
                        int max_pages, const int* __restrict__ seq_starts, const int* __restrict__ positions, int page_size, int H, int L,
                        int R, float scale, __nv_bfloat16* __restrict__ out, long o_ts, long o_hs, int WPH, int colsw, int window,
                        const int* __restrict__ row_seq, int splits, float* __restrict__ part) {
    constexpr int BN = VOB_LTC_BN;
    constexpr int PRE = HEADS && NT16 <= 4 ? 5 : VOB_LTC_PRE;       // two blocks an SM leave room for fewer
    pdl_launch_dependents();
    pdl_wait(48);
    const int NW = blockDim.x >> 5, HB = NW / WPH;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int hh = warp / WPH, wsub = warp - hh * WPH;
    const int h = (blockIdx.y * HB + hh) * (HEADS ? 16 : 1);       // this warp's head, or the first of its 16 heads
    const bool head = h < H;
    int s, r0, nrows;
    if (HEADS) {
        r0 = blockIdx.x;
        s = row_seq[r0];
        nrows = max(0, min(16, H - h));
        if (positions[r0] < 0) {                                   // padding: nothing to see
            for (int i = lane; head && wsub == 0 && i < nrows * L; i += 32) {
                if (splits == 1) out[(size_t)r0 * o_ts + (size_t)(h + i / L) * o_hs + i % L] = __float2bfloat16_rn(0.f);
            }
            return;                                                // (the merge writes zeros for such rows by itself)
        }
    } else {
        s = blockIdx.z;
        const int r1 = seq_starts[s + 1];
        r0 = seq_starts[s] + blockIdx.x * 16;
        if (r0 >= r1) return;
        nrows = min(16, r1 - r0);
    }
    const int D = L + R, DP = D + 8;
    extern __shared__ __align__(128) unsigned char ltc_smem[];
    __nv_bfloat16* Kt = reinterpret_cast<__nv_bfloat16*>(ltc_smem);                               // [BN][DP]
    __nv_bfloat16* Q = Kt + (size_t)BN * DP + (size_t)hh * 16 * DP;                                // [16][DP] per head
    // the queries, rounded: four features a lane, up to four rows of a warp in flight (L and R are multiples of 16)
    for (int i0 = wsub; i0 < 16; i0 += 4 * WPH) {
        for (int c = 4 * lane; c < D; c += 128) {
            float4 v[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int i = i0 + k * WPH;
                v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (head && i < nrows) {
                    const size_t tok = HEADS ? r0 : r0 + i, hd = HEADS ? h + i : h;
                    v[k] = *reinterpret_cast<const float4*>(c < L ? q_lat + tok * q_ts + hd * q_hs + c : q_rot + (tok * H + hd) * R + (c - L));
                }
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int i = i0 + k * WPH;
                if (i < 16) *reinterpret_cast<uint2*>(Q + i * DP + c) = make_uint2(pack_bf16(v[k].x, v[k].y), pack_bf16(v[k].z, v[k].w));
            }
        }
    }
    const int pos0 = positions[r0];
    int pos_hi = HEADS ? pos0 : pos0 + nrows - 1;
    // with a window a row sees only its last `window` keys: the tile's first row bounds the keys from below (pages before
    // that may have been given back and are never addressed), and the walk starts at the tile of BN keys that holds it, so
    // that a row's keys fall into the same tiles however the prompt was cut
    const int key_lo = window > 0 ? max(0, pos0 + 1 - window) : 0;
    int k_start = key_lo / BN * BN;
    if (HEADS) {                                   // this block's share of the tiles
        const int tiles = (pos0 - k_start) / BN + 1, per = (tiles + splits - 1) / splits;
        k_start += (int)blockIdx.z * per * BN;
        pos_hi = min(pos0, k_start + per * BN - 1);
    }
    const int* table = block_tables + (size_t)s * max_pages;
    // this warp's latent columns, in groups of 16
    const int col0 = wsub * colsw;
    const int n16 = max(0, min(colsw, L - col0)) / 16;
    const int g = lane >> 2, t4 = lane & 3;          // this thread's rows g and g + 8, columns 2 * t4, + 1 of every 8
    float o[NT16 * 2][4];
#pragma unroll
    for (int i = 0; i < NT16 * 2; ++i) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;       // l: this thread's share of the row sums
    const bool row0 = g < nrows, row1 = g + 8 < nrows;
    const int p0 = HEADS ? pos0 : pos0 + g, p1 = HEADS ? pos0 : pos0 + g + 8;       // these rows' positions
    const int lat_chunks = L / 8, kr_chunks = R / 8;            // 16-byte pieces of a key
    // The key tile as a list of 16-byte pieces, BN keys x (lat_chunks + kr_chunks) pieces: thread t takes pieces
    // t, t + threads, ... The NEXT tile's pieces are fetched into registers while this tile is worked on.
    const int pieces = lat_chunks + kr_chunks, tile_pieces = BN * pieces;
    const int dp_pieces = DP / 8;                    // a row of Kt in 16-byte pieces (DP is a multiple of 8)
    uint4 nxt[PRE];
    // where this thread's pieces lie in a tile, the same in every tile: key << 8 | piece, two to a register
    unsigned place[(PRE + 1) / 2];
#pragma unroll
    for (int i = 0; i < PRE; ++i) {
        const int x = (int)threadIdx.x + i * (int)blockDim.x;
        const unsigned kk = x / pieces, pc = (kk << 8) | (unsigned)(x - (int)kk * pieces);
        if (i & 1) place[i >> 1] |= pc << 16;
        else place[i >> 1] = pc & 0xffffu;
    }
    const int shift = (page_size & (page_size - 1)) == 0 ? 31 - __clz(page_size) : -1;       // pages of a power of two: no division
    auto piece = [&](int key, int c) {
        uint4 val = make_uint4(0u, 0u, 0u, 0u);
        if (key <= pos_hi && key >= key_lo) {
            const int pg = shift >= 0 ? key >> shift : key / page_size;
            const size_t slot = (size_t)table[pg] * page_size + (key - pg * page_size);
            val = c < lat_chunks ? reinterpret_cast<const uint4*>(lat + slot * L)[c] : reinterpret_cast<const uint4*>(kr + slot * R)[c - lat_chunks];
        }
        return val;
    };
    auto fetch = [&](int k0) {
#pragma unroll
        for (int i = 0; i < PRE; ++i) {
            const unsigned pc = i & 1 ? place[i >> 1] >> 16 : place[i >> 1] & 0xffffu;
            if ((int)threadIdx.x + i * (int)blockDim.x < tile_pieces) nxt[i] = piece(k0 + (int)(pc >> 8), (int)(pc & 255u));
        }
    };
    fetch(k_start);
    const float scale2 = scale * 1.4426950408889634f;        // scores in units of ln 2, for exp2f
    const int p_min = pos0, p_max = HEADS ? pos0 : pos0 + nrows - 1;             // positions of the tile's first and last row
    for (int k0 = k_start; k0 <= pos_hi; k0 += BN) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < PRE; ++i) {
            const unsigned pc = i & 1 ? place[i >> 1] >> 16 : place[i >> 1] & 0xffffu;
            if ((int)threadIdx.x + i * (int)blockDim.x < tile_pieces)
                reinterpret_cast<uint4*>(Kt)[(pc >> 8) * (unsigned)dp_pieces + (pc & 255u)] = nxt[i];
        }
        // what of a tile the registers do not hold (small blocks, wide keys) is copied now
        for (int x = (int)threadIdx.x + PRE * (int)blockDim.x; x < tile_pieces; x += (int)blockDim.x) {
            const int kk = x / pieces, c = x - kk * pieces;
            reinterpret_cast<uint4*>(Kt)[(size_t)kk * dp_pieces + c] = piece(k0 + kk, c);
        }
        if (k0 + BN <= pos_hi) fetch(k0 + BN);
        __syncthreads();
        if (!head) continue;
        // S = Q K^T: 16 rows x 32 keys, four accumulator tiles of 8 keys
        float sc[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) { sc[j][0] = 0.f; sc[j][1] = 0.f; sc[j][2] = 0.f; sc[j][3] = 0.f; }
#pragma unroll 2
        for (int ks = 0; ks < D / 16; ++ks) {
            unsigned a0, a1, a2, a3;
            ldsm_x4(a0, a1, a2, a3, Q + (size_t)(lane & 15) * DP + ks * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int jp = 0; jp < 2; ++jp) {            // keys 16 * jp .. + 15: two accumulator tiles
                unsigned b0, b1, b2, b3;
                ldsm_x4(b0, b1, b2, b3, Kt + (size_t)(16 * jp + (lane >> 4) * 8 + (lane & 7)) * DP + ks * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16_16816(sc[2 * jp], a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(sc[2 * jp + 1], a0, a1, a2, a3, b2, b3);
            }
        }
        // the softmax of rows g and g + 8 over this tile's keys
        float mx0 = -INFINITY, mx1 = -INFINITY;
        if (k0 + BN - 1 <= p_min && (window <= 0 || k0 > p_max - window)) {      // every row sees the whole tile
#pragma unroll
            for (int j = 0; j < 4; ++j) {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    sc[j][e] *= scale2;
                    sc[j][2 + e] *= scale2;
                    mx0 = fmaxf(mx0, sc[j][e]);
                    mx1 = fmaxf(mx1, sc[j][2 + e]);
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int key = k0 + 8 * j + 2 * t4 + e;
                    const bool in0 = key <= p0 && (window <= 0 || key > p0 - window);
                    const bool in1 = key <= p1 && (window <= 0 || key > p1 - window);
                    sc[j][e] = (row0 && in0) ? sc[j][e] * scale2 : -INFINITY;
                    sc[j][2 + e] = (row1 && in1) ? sc[j][2 + e] * scale2 : -INFINITY;
                    mx0 = fmaxf(mx0, sc[j][e]);
                    mx1 = fmaxf(mx1, sc[j][2 + e]);
                }
            }
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
        const bool none0 = mn0 == -INFINITY, none1 = mn1 == -INFINITY;
        const float corr0 = none0 ? 1.f : exp2f(m0 - mn0), corr1 = none1 ? 1.f : exp2f(m1 - mn1);
        float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                sc[j][e] = none0 ? 0.f : exp2f(sc[j][e] - mn0);
                sc[j][2 + e] = none1 ? 0.f : exp2f(sc[j][2 + e] - mn1);
                sum0 += sc[j][e];
                sum1 += sc[j][2 + e];
            }
        }
        l0 = fmaf(l0, corr0, sum0);
        l1 = fmaf(l1, corr1, sum1);
        m0 = mn0;
        m1 = mn1;
        // P as the A operand of the second product: the accumulator tiles of 8 keys pair up into 16 keys
        unsigned pa[2][4];
#pragma unroll
        for (int jp = 0; jp < 2; ++jp) {
            pa[jp][0] = pack_bf16(sc[2 * jp][0], sc[2 * jp][1]);
            pa[jp][1] = pack_bf16(sc[2 * jp][2], sc[2 * jp][3]);
            pa[jp][2] = pack_bf16(sc[2 * jp + 1][0], sc[2 * jp + 1][1]);
            pa[jp][3] = pack_bf16(sc[2 * jp + 1][2], sc[2 * jp + 1][3]);
        }
        // O = O * corr + P C over this warp's latent columns
#pragma unroll
        for (int n = 0; n < NT16; ++n) {
            if (n < n16) {
                o[2 * n][0] *= corr0; o[2 * n][1] *= corr0; o[2 * n][2] *= corr1; o[2 * n][3] *= corr1;
                o[2 * n + 1][0] *= corr0; o[2 * n + 1][1] *= corr0; o[2 * n + 1][2] *= corr1; o[2 * n + 1][3] *= corr1;
#pragma unroll
                for (int jp = 0; jp < 2; ++jp) {
                    unsigned b0, b1, b2, b3;
                    ldsm_x4_trans(b0, b1, b2, b3, Kt + (size_t)(16 * jp + ((lane >> 3) & 1) * 8 + (lane & 7)) * DP + col0 + 16 * n + (lane >> 4) * 8);
                    mma_bf16_16816(o[2 * n], pa[jp][0], pa[jp][1], pa[jp][2], pa[jp][3], b0, b1);
                    mma_bf16_16816(o[2 * n + 1], pa[jp][0], pa[jp][1], pa[jp][2], pa[jp][3], b2, b3);
                }
            }
        }
    }
    if (!head) return;
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    if (HEADS && splits > 1) {                     // (maximum, sum, weighted sum) of this share, per head
        float* pr0 = part + (((size_t)r0 * H + h + g) * splits + blockIdx.z) * (L + 2);
        float* pr1 = pr0 + (size_t)8 * splits * (L + 2);
        if (wsub == 0 && t4 == 0) {
            if (row0) { pr0[0] = m0 * 0.6931471805599453f; pr0[1] = l0; }
            if (row1) { pr1[0] = m1 * 0.6931471805599453f; pr1[1] = l1; }
        }
#pragma unroll
        for (int n = 0; n < NT16 * 2; ++n) {
            if (n < 2 * n16) {
                const int c = 2 + col0 + 8 * n + 2 * t4;          // L + 2 is even: pairs of columns are 8-byte aligned
                if (row0) *reinterpret_cast<float2*>(pr0 + c) = make_float2(o[n][0], o[n][1]);
                if (row1) *reinterpret_cast<float2*>(pr1 + c) = make_float2(o[n][2], o[n][3]);
            }
        }
        return;
    }
    const float inv0 = 1.0f / l0, inv1 = 1.0f / l1;
    __nv_bfloat16* o0 = out + (size_t)(HEADS ? r0 : r0 + g) * o_ts + (size_t)(HEADS ? h + g : h) * o_hs;
    __nv_bfloat16* o1 = o0 + (HEADS ? 8 * o_hs : 8 * o_ts);
#pragma unroll
    for (int n = 0; n < NT16 * 2; ++n) {
        if (n < 2 * n16) {
            const int c = col0 + 8 * n + 2 * t4;
            if (row0) *reinterpret_cast<__nv_bfloat162*>(o0 + c) = __floats2bfloat162_rn(o[n][0] * inv0, o[n][1] * inv0);
            if (row1) *reinterpret_cast<__nv_bfloat162*>(o1 + c) = __floats2bfloat162_rn(o[n][2] * inv1, o[n][3] * inv1);
        }
    }
}

// The shape of a block of the tensor-core kernel: warps per head (each with at most 256 latent columns, a multiple of
// 16), the columns per warp, and heads per block (0: the sizes do not fit the kernel).
static int ltc_shape(int H, int L, int R, int* wph, int* colsw) {
    if (L % 16 || R % 16 || L <= 0 || R <= 0 || L > 1024) return 0;
    *wph = (L + 255) / 256;
    *colsw = ((L / 16 + *wph - 1) / *wph) * 16;
    const size_t DP = (size_t)L + R + 8;
    const size_t shared = (size_t)VOB_LTC_BN * DP * 2, per_head = 16 * DP * 2;
    int hb = 8 / *wph;                                   // at most eight warps
    while (hb > 1 && shared + hb * per_head > 100 * 1024) --hb;
    if (shared + hb * per_head > 200 * 1024) return 0;
    return hb > H ? H : hb;
}

VOB_EXPORT int vob_latent_attend_tc_supported(int H, int L, int R) {
    int wph, colsw;
    return ltc_shape(H, L, R, &wph, &colsw) > 0 ? 1 : 0;
}

// q_lat, q_rot, out and the caches as for vob_latent_attend (bfloat16 caches and out only; out's strides even);
// seq_starts int32 [seqs + 1]; max_new: no request brings more rows than this.
VOB_EXPORT int vob_latent_attend_tc(const float* q_lat, long q_ts, long q_hs, const float* q_rot, const void* lat, const void* kr,
                                    const int* block_tables, int max_pages, const int* seq_starts, const int* positions, int page_size,
                                    int seqs, int max_new, int H, int L, int R, float scale, void* out, long o_ts, long o_hs,
                                    int window, cudaStream_t stream) {
    if (seqs <= 0 || max_new <= 0) return 0;
    if (window < 0) return VOB_ERR_BAD_ARG;
    int wph, colsw;
    const int hb = ltc_shape(H, L, R, &wph, &colsw);
    if (hb <= 0) return VOB_ERR_UNSUPPORTED;
    if (page_size <= 0 || max_pages <= 0 || seqs > 65535 || (H + hb - 1) / hb > 65535 || (o_ts & 1) || (o_hs & 1) || ((uintptr_t)out & 3)
        || (q_ts & 3) || (q_hs & 3) || (((uintptr_t)q_lat | (uintptr_t)q_rot) & 15))
        return VOB_ERR_BAD_ARG;
    const size_t DP = (size_t)L + R + 8;
    const size_t smem = (size_t)VOB_LTC_BN * DP * 2 + (size_t)hb * 16 * DP * 2;
    dim3 grid((max_new + 15) / 16, (H + hb - 1) / hb, seqs), block(32 * hb * wph);
#define VOB_LTC(N)                                                                                                              \
    do {                                                                                                                        \
        cudaError_t e = cudaFuncSetAttribute(latent_attend_tc_kernel<N, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e != cudaSuccess) return (int)e;                                                                                    \
        return vob_launch(latent_attend_tc_kernel<N, false>, grid, block, smem, stream, q_lat, q_ts, q_hs, q_rot, (const __nv_bfloat16*)lat, \
                          (const __nv_bfloat16*)kr, block_tables, max_pages, seq_starts, positions, page_size, H, L, R, scale,  \
                          (__nv_bfloat16*)out, o_ts, o_hs, wph, colsw, window, nullptr, 1, nullptr);                            \
    } while (0)
    if (colsw <= 64) VOB_LTC(4);
    if (colsw <= 128) VOB_LTC(8);
    VOB_LTC(16);
#undef VOB_LTC
}


// The shape of a block in steps of single tokens: groups of 16 heads per block, and the warps that share a group's latent columns.
static int ltc_heads_shape(int H, int L, int R, int* wph, int* colsw) {
    if (L % 16 || R % 16 || L <= 0 || R <= 0 || L > 1024 || H <= 0) return 0;
    const size_t DP = (size_t)L + R + 8;
    const size_t shared = (size_t)VOB_LTC_BN * DP * 2, per_group = 16 * DP * 2;
    const int least = (L + 255) / 256, groups = (H + 15) / 16;
    int hb = groups < 4 ? groups : 4;
    while (hb > 1 && (shared + hb * per_group > 100 * 1024 || hb * least > 8)) --hb;
    if (shared + hb * per_group > 200 * 1024) return 0;
    int w = 8 / hb;
    if (w > L / 16) w = L / 16;
    *wph = w < least ? least : w;
    *colsw = ((L / 16 + *wph - 1) / *wph) * 16;
    return hb;
}

// Groups of 16 heads a block takes, 0: the sizes do not fit.
VOB_EXPORT int vob_latent_decode_tc_groups(int H, int L, int R) {
    int wph, colsw;
    return ltc_heads_shape(H, L, R, &wph, &colsw);
}

// Steps of single tokens: row t is one token of request row_seq[t]. Operands as for vob_latent_attend (bfloat16 caches and out
// only; out's strides even, part 8-byte aligned).
VOB_EXPORT int vob_latent_decode_tc(const float* q_lat, long q_ts, long q_hs, const float* q_rot, const void* lat, const void* kr,
                                    const int* block_tables, int max_pages, const int* row_seq, const int* positions, int page_size, int T,
                                    int H, int L, int R, float scale, void* out, long o_ts, long o_hs, int splits, float* part, int window,
                                    cudaStream_t stream) {
    if (T <= 0) return 0;
    int wph, colsw;
    const int hb = ltc_heads_shape(H, L, R, &wph, &colsw);
    if (hb <= 0) return VOB_ERR_UNSUPPORTED;
    if (window < 0 || page_size <= 0 || max_pages <= 0 || splits < 1 || splits > VOB_LATENT_SPLITS || (splits > 1 && !part) || H > 65535
        || (o_ts & 1) || (o_hs & 1) || ((uintptr_t)out & 3) || ((uintptr_t)part & 7)
        || (q_ts & 3) || (q_hs & 3) || (((uintptr_t)q_lat | (uintptr_t)q_rot) & 15))
        return VOB_ERR_BAD_ARG;
    const size_t DP = (size_t)L + R + 8;
    const size_t smem = (size_t)VOB_LTC_BN * DP * 2 + (size_t)hb * 16 * DP * 2;
    dim3 grid(T, ((H + 15) / 16 + hb - 1) / hb, splits), block(32 * hb * wph);
    int status = VOB_ERR_BAD_ARG;
#define VOB_LTCH(N)                                                                                                                   \
    do {                                                                                                                              \
        cudaError_t e = cudaFuncSetAttribute(latent_attend_tc_kernel<N, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e != cudaSuccess) return (int)e;                                                                                          \
        status = vob_launch(latent_attend_tc_kernel<N, true>, grid, block, smem, stream, q_lat, q_ts, q_hs, q_rot, (const __nv_bfloat16*)lat, \
                            (const __nv_bfloat16*)kr, block_tables, max_pages, nullptr, positions, page_size, H, L, R, scale,          \
                            (__nv_bfloat16*)out, o_ts, o_hs, wph, colsw, window, row_seq, splits, part);                              \
    } while (0)
    if (colsw <= 64) VOB_LTCH(4);
    else if (colsw <= 128) VOB_LTCH(8);
    else VOB_LTCH(16);
#undef VOB_LTCH
    if (status == 0 && splits > 1)
        status = vob_launch(latent_merge_kernel<__nv_bfloat16>, dim3(T, H), dim3(128), 0, stream, (const float*)part, positions, H, L, splits,
                            (__nv_bfloat16*)out, o_ts, o_hs);
    return status;
}
