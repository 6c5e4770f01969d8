// layered_mixers4.cuh -- more mechanisms of the layered runtime (layered.cu), under the rules of layered_kernels.cuh: a kernel per
// mechanism, constants as arguments, fp32 for everything that is not a matrix-product operand, positions optionally read from a device
// word (captured decode step).
//
//   output norms         k_post_norm (a sublayer is normed on its way out only: x += unit(y) w, where y is one branch or the weighted
//                        sum of two branches, each with a norm of its own)
//   attention            k_qk_norm_rope (query and key norm over the whole projection, "rotate half" positions, keys and values into the
//                        cache pages), k_gqa_attn (grouped-query causal softmax attention for long portions: the query heads of a
//                        key/value head are rows of one register-tiled product; soft cap, sink, one sigmoid gate per head),
//                        k_gqa_decode (the same for short portions: norm, rotation, cache write, scores, softmax and merge of the key
//                        splits in one launch)
//   gated delta rule     per head  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q,  g one number or one per key channel.
//                        k_delta_prep (convolution, silu, unit vectors, step size, decay, and everything that lets kDeltaChunk tokens be
//                        solved together), k_delta_scan (the recurrence of a long portion, kDeltaChunk tokens per step), k_delta_step
//                        (short portions: everything after the convolution up to the gated, normed output, a cluster of blocks per head)
#pragma once
#include "layered_mixers3.cuh"

namespace nb {
namespace lm {

// ------------------------------------------------------------------------------------------------
// x[t] += y / rms(y) w  with  y = d[t],  or (d2 given)  y = mix (d / rms(d) w1 + d2 / rms(d2) w2);  keep (optional) receives the updated x.
// One block per token; NV > 0: a thread keeps its (at most NV) elements in registers between the reductions.
// ------------------------------------------------------------------------------------------------
struct PostNormArgs { float *x; const float *d, *d2; const float *w1, *w2, *w; float mix; float *keep; uint32_t T, E; float eps; };
// two sums over the block at once
__device__ __forceinline__ float2 block_sum2(float2 v, float2 *red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) { v.x += __shfl_xor_sync(0xffffffffu, v.x, o); v.y += __shfl_xor_sync(0xffffffffu, v.y, o); }
    __syncthreads();
    if ((threadIdx.x & 31u) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float2 s = make_float2(0.0f, 0.0f);
    for (uint32_t w = 0; w < (blockDim.x >> 5); w++) { s.x += red[w].x; s.y += red[w].y; }
    return s;
}
template <int NV>
__global__ void __launch_bounds__(1024) k_post_norm(const PostNormArgs a) {
    pdl_enter();
    __shared__ float2 red[32];
    const size_t row = (size_t)blockIdx.x * a.E;
    const float *d = a.d + row, *d2 = a.d2 ? a.d2 + row : nullptr;
    float *x = a.x + row;
    float y[NV > 0 ? NV : 1], z[NV > 0 ? NV : 1], xv[NV > 0 ? NV : 1];
    float2 s = make_float2(0.0f, 0.0f);
    if constexpr (NV > 0) {
#pragma unroll
        for (int k = 0; k < NV; k++) {
            const uint32_t i = threadIdx.x + k * blockDim.x;
            const bool ok = i < a.E;
            y[k] = ok ? d[i] : 0.0f; z[k] = (ok && d2) ? d2[i] : 0.0f; xv[k] = ok ? x[i] : 0.0f;
            s.x = fmaf(y[k], y[k], s.x); s.y = fmaf(z[k], z[k], s.y);
        }
    } else {
        for (uint32_t i = threadIdx.x; i < a.E; i += blockDim.x) { const float u = d[i], v = d2 ? d2[i] : 0.0f; s.x = fmaf(u, u, s.x); s.y = fmaf(v, v, s.y); }
    }
    s = block_sum2(s, red);
    float rinv = 1.0f / sqrtf(s.x / (float)a.E + a.eps);
    const float ra = rinv, rb = 1.0f / sqrtf(s.y / (float)a.E + a.eps);
    if (d2) {
        s = make_float2(0.0f, 0.0f);
        if constexpr (NV > 0) {
#pragma unroll
            for (int k = 0; k < NV; k++) {
                const uint32_t i = threadIdx.x + k * blockDim.x;
                y[k] = i < a.E ? a.mix * (y[k] * ra * a.w1[i] + z[k] * rb * a.w2[i]) : 0.0f;
                s.x = fmaf(y[k], y[k], s.x);
            }
        } else {
            for (uint32_t i = threadIdx.x; i < a.E; i += blockDim.x) { const float u = a.mix * (d[i] * ra * a.w1[i] + d2[i] * rb * a.w2[i]); s.x = fmaf(u, u, s.x); }
        }
        s = block_sum2(s, red);
        rinv = 1.0f / sqrtf(s.x / (float)a.E + a.eps);
    }
    if constexpr (NV > 0) {
#pragma unroll
        for (int k = 0; k < NV; k++) {
            const uint32_t i = threadIdx.x + k * blockDim.x;
            if (i >= a.E) continue;
            const float v = xv[k] + y[k] * rinv * a.w[i];
            x[i] = v;
            if (a.keep) a.keep[row + i] = v;
        }
    } else
    for (uint32_t i = threadIdx.x; i < a.E; i += blockDim.x) {
        const float u = d2 ? a.mix * (d[i] * ra * a.w1[i] + d2[i] * rb * a.w2[i]) : d[i];
        const float v = x[i] + u * rinv * a.w[i];
        x[i] = v;
        if (a.keep) a.keep[row + i] = v;
    }
}

// ------------------------------------------------------------------------------------------------
// Grouped-query attention.  Rows of the joint product hold q [H][D] at q0, k [G][D] at k0, v [G][VD] at v0 and one gate number per head
// at g0.  wq / wk (optional): gains of an RMS norm over ALL rows of q (of k) at once, or (head_norm) over every head by itself, D gains
// shared by the heads.  block (0: none): a query sees the keys of its own block of that many positions only, counted from position 0.  tab (optional): (cos, sin)[position][half];
// coordinate i < half turns with i + half, (u, v) -> (u cos - v sin, v cos + u sin); the rest of a head passes.  q carries the score
// scale afterwards.  A cache row is [G D keys | G VD values | padding to 4].
// ------------------------------------------------------------------------------------------------
struct GqaArgs {
    float *p; uint32_t ld, q0, k0, v0, g0; const float *wq, *wk; const float2 *tab; uint32_t half;
    float *cache; const uint32_t *table; uint32_t T, H, G, D, VD, RL, pos0; const uint32_t *pos_ptr; float eps;
    float scale, softcap; const float *sink; uint32_t has_gate; float *out;      // softcap 0: none; sink null: none; out [T][H VD]
    uint32_t nsplit; float *part; uint32_t *tickets; uint32_t hb;                // k_gqa_decode: key splits; query heads per block
    uint32_t block, head_norm;
};
__device__ __forceinline__ uint32_t gqa_first(uint32_t pos, uint32_t block) { return block ? pos - pos % block : 0u; }      // the first key position pos sees
// coordinate d of one head: normed by r and its gains, turned
__device__ __forceinline__ float rot_half_at(const float *x, const float *w, float r, uint32_t d, uint32_t half, const float2 *cs) {
    const float u = x[d] * r * (w ? w[d] : 1.0f);
    if (d >= 2u * half) return u;
    const uint32_t i = d < half ? d : d - half, o = d < half ? d + half : i;
    const float v = x[o] * r * (w ? w[o] : 1.0f);
    const float2 c = cs[i];
    return d < half ? u * c.x - v * c.y : u * c.x + v * c.y;
}
__global__ void __launch_bounds__(256) k_qk_norm_rope(const GqaArgs a) {
    pdl_enter();
    __shared__ float2 red[32];
    const uint32_t t = blockIdx.x, pos = a.pos0 + t + (a.pos_ptr ? *a.pos_ptr : 0u), QW = a.H * a.D, KW = a.G * a.D, half = a.tab ? a.half : 0u;
    float *q = a.p + (size_t)t * a.ld + a.q0;
    const float *k = a.p + (size_t)t * a.ld + a.k0, *v = a.p + (size_t)t * a.ld + a.v0;
    float rq = 1.0f, rk = 1.0f;
    if ((a.wq || a.wk) && !a.head_norm) {
        float2 s = make_float2(0.0f, 0.0f);
        for (uint32_t i = threadIdx.x; i < QW; i += blockDim.x) s.x = fmaf(q[i], q[i], s.x);
        for (uint32_t i = threadIdx.x; i < KW; i += blockDim.x) s.y = fmaf(k[i], k[i], s.y);
        s = block_sum2(s, red);
        if (a.wq) rq = 1.0f / sqrtf(s.x / (float)QW + a.eps);
        if (a.wk) rk = 1.0f / sqrtf(s.y / (float)KW + a.eps);
    }
    const float2 *cs = a.tab + (size_t)pos * half;
    // a warp per head; q in place (a lane owns both coordinates of a pair), k into the token's cache row, v beside it
    const uint32_t per = a.D - half, warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, nw = blockDim.x >> 5;
    float *row = a.cache + ((size_t)a.table[pos / kPage] * kPage + pos % kPage) * a.RL;
    for (uint32_t h = warp; h < a.H + a.G; h += nw) {
        const bool isq = h < a.H;
        const uint32_t hh = (isq ? h : h - a.H) * a.D;
        const float *src = (isq ? q : k) + hh, *w = isq ? a.wq : a.wk;
        float *dst = isq ? q + hh : row + hh;
        float r = isq ? rq * a.scale : rk;
        if (a.head_norm && w) {
            float s = 0.0f;
            for (uint32_t e = lane; e < a.D; e += 32u) s = fmaf(src[e], src[e], s);
            r *= 1.0f / sqrtf(warp_sum(s) / (float)a.D + a.eps);
        } else if (w) w += hh;
        for (uint32_t e = lane; e < per; e += 32u) {
            if (e < half) {
                const float u = src[e] * r * (w ? w[e] : 1.0f), z = src[e + half] * r * (w ? w[e + half] : 1.0f);
                const float2 c = cs[e];
                dst[e] = u * c.x - z * c.y; dst[e + half] = z * c.x + u * c.y;
            } else dst[e + half] = src[e + half] * r * (w ? w[e + half] : 1.0f);
        }
    }
    for (uint32_t i = threadIdx.x; i < a.RL - KW; i += blockDim.x) row[KW + i] = i < a.G * a.VD ? v[i] : 0.0f;
}

// Long portions.  Row r of key/value head g is query token r / rep, query head g rep + r % rep (rep = H / G): all heads that share keys
// share a block, which multiplies 64 rows with 64 keys (two cache pages) at a time -- scores in a 4 x 4 register tile per thread, the
// weighted sum in a 4 x (4 VJ) tile.  The sink is the softmax's first term: m = sink, l = 1, no value.  q must have passed
// k_qk_norm_rope.  grid = (row tiles, G); 256 threads.
constexpr uint32_t kGqaM = 64, kGqaN = 64;
__host__ __device__ inline uint32_t gqa_ld(uint32_t D) { const uint32_t Dp = (D + 3u) & ~3u; return ((Dp >> 2) & 1u) ? Dp : Dp + 4u; }      // rows of an odd number of 16-byte units
__host__ __device__ inline uint32_t gqa_kwords(uint32_t D) { const uint32_t k = kGqaN * gqa_ld(D), p = kGqaM * (kGqaN + 4u); return k > p ? k : p; }
inline size_t gqa_attn_smem(uint32_t D, int vj) { return ((size_t)kGqaM * gqa_ld(D) + gqa_kwords(D) + (size_t)kGqaN * vj * 64u) * 4; }
__device__ __forceinline__ void cp_async16(float *dst, const float *src, bool ok) {      // 16 bytes into shared memory; zeros when !ok
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst), n = ok ? 16u : 0u;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }
template <int VJ>
__global__ void __launch_bounds__(256, VJ <= 2 ? 2 : 1) k_gqa_attn(const GqaArgs a) {
    pdl_enter();
    extern __shared__ __align__(16) float sm[];
    const uint32_t D = a.D, VD = a.VD, Dp = (D + 3u) & ~3u, LD = gqa_ld(D), D4 = Dp / 4u, rep = a.H / a.G, rows = a.T * rep, g = blockIdx.y;
    constexpr uint32_t LDP = kGqaN + 4u, LDV = VJ * 64u;
    float *q_s = sm, *k_s = q_s + kGqaM * LD, *v_s = k_s + gqa_kwords(D), *p_s = k_s;      // the weights take the keys' place once the scores are made
    const uint32_t tid = threadIdx.x, ty = tid >> 4, tx = tid & 15u;
    const uint32_t r0 = (gridDim.x - 1u - blockIdx.x) * kGqaM;            // the longest tiles first
    const uint32_t pos = a.pos0 + (a.pos_ptr ? *a.pos_ptr : 0u);
    const uint32_t t_last = (min(rows, r0 + kGqaM) - 1u) / rep, nkeys = pos + t_last + 1u, tiles = (nkeys + kGqaN - 1u) / kGqaN, tile0 = gqa_first(pos + r0 / rep, a.block) / kGqaN;
    const bool vec = ((D | VD | a.ld | a.q0) & 3u) == 0;
    for (uint32_t i = tid; i < kGqaM * D4; i += 256u) {
        const uint32_t r = i / D4, d = (i % D4) * 4u, rr = r0 + r;
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (rr < rows) {
            const float *src = a.p + (size_t)(rr / rep) * a.ld + a.q0 + (g * rep + rr % rep) * D + d;
            if (vec) v = *reinterpret_cast<const float4 *>(src);
            else { v.x = src[0]; if (d + 1u < D) v.y = src[1]; if (d + 2u < D) v.z = src[2]; if (d + 3u < D) v.w = src[3]; }
        }
        *reinterpret_cast<float4 *>(q_s + r * LD + d) = v;
    }
    float m[4], l[4], o[4][VJ * 4];
    uint32_t lim[4], low[4];               // the last and the first key each of this thread's rows sees
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t rr = min(r0 + ty * 4u + i, rows - 1u);
        lim[i] = pos + rr / rep; low[i] = gqa_first(lim[i], a.block);
        m[i] = a.sink ? a.sink[g * rep + rr % rep] : -INFINITY; l[i] = a.sink ? 1.0f : 0.0f;
#pragma unroll
        for (int c = 0; c < VJ * 4; c++) o[i][c] = 0.0f;
    }
    for (uint32_t tile = tile0; tile < tiles; tile++) {
        __syncthreads();
        const uint32_t key0 = tile * kGqaN;
        // both pages of the tile; keys past the block's last one become zeros
        const float *pg0 = a.cache + (size_t)a.table[key0 / kPage] * kPage * a.RL;
        const float *pg1 = key0 + kPage < nkeys ? a.cache + (size_t)a.table[key0 / kPage + 1u] * kPage * a.RL : pg0;
        if (vec) {
            const uint32_t w4 = D4 + VD / 4u;
            for (uint32_t i = tid; i < kGqaN * w4; i += 256u) {
                const uint32_t k = i / w4, e = i % w4;
                const float *row = (k < kPage ? pg0 : pg1) + (size_t)(k % kPage) * a.RL;
                const bool ok = key0 + k < nkeys;
                if (e < D4) cp_async16(k_s + k * LD + e * 4u, row + g * D + e * 4u, ok);
                else cp_async16(v_s + k * LDV + (e - D4) * 4u, row + a.G * D + g * VD + (e - D4) * 4u, ok);
            }
            cp_async_wait();
        } else {
            for (uint32_t i = tid; i < kGqaN * (Dp + VD); i += 256u) {
                const uint32_t k = i / (Dp + VD), e = i % (Dp + VD);
                const float *row = (k < kPage ? pg0 : pg1) + (size_t)(k % kPage) * a.RL;
                const bool ok = key0 + k < nkeys;
                if (e < Dp) k_s[k * LD + e] = (ok && e < D) ? row[g * D + e] : 0.0f;
                else v_s[k * LDV + e - Dp] = ok ? row[a.G * D + g * VD + e - Dp] : 0.0f;
            }
        }
        __syncthreads();
        float s[4][4] = {};
#pragma unroll 2
        for (uint32_t e = 0; e < D4; e++) {
            float4 qv[4], kv[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { qv[i] = *reinterpret_cast<const float4 *>(q_s + (ty * 4u + i) * LD + e * 4u); kv[i] = *reinterpret_cast<const float4 *>(k_s + (tx + 16u * i) * LD + e * 4u); }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) s[i][j] = fmaf(qv[i].w, kv[j].w, fmaf(qv[i].z, kv[j].z, fmaf(qv[i].y, kv[j].y, fmaf(qv[i].x, kv[j].x, s[i][j]))));
        }
        __syncthreads();                   // every key of the tile has been read: the weights may take its place
#pragma unroll
        for (int i = 0; i < 4; i++) {
            float tm = -INFINITY;
#pragma unroll
            for (int j = 0; j < 4; j++) {
                float v = s[i][j];
                if (a.softcap > 0.0f) v = a.softcap * tanhf(v / a.softcap);
                s[i][j] = key0 + tx + 16u * j <= lim[i] && key0 + tx + 16u * j >= low[i] ? v : -INFINITY;
                tm = fmaxf(tm, s[i][j]);
            }
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, off));
            const float mn = fmaxf(m[i], tm), corr = mn == -INFINITY ? 1.0f : expf(m[i] - mn);
            float ps = 0.0f;
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const float pv = s[i][j] == -INFINITY ? 0.0f : expf(s[i][j] - mn);
                p_s[(ty * 4u + i) * LDP + tx + 16u * j] = pv;
                ps += pv;
            }
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, off);
            l[i] = fmaf(l[i], corr, ps);
            m[i] = mn;
#pragma unroll
            for (int c = 0; c < VJ * 4; c++) o[i][c] *= corr;
        }
        __syncwarp();                      // a row's 16 threads sit in one warp: its weights are read by the warp that wrote them
#pragma unroll 1
        for (uint32_t k = 0; k < kGqaN; k += 4u) {
            float4 pv[4];
#pragma unroll
            for (int i = 0; i < 4; i++) pv[i] = *reinterpret_cast<const float4 *>(p_s + (ty * 4u + i) * LDP + k);
#pragma unroll
            for (int kk = 0; kk < 4; kk++)
#pragma unroll
                for (int j = 0; j < VJ; j++) {
                    const float4 vv = *reinterpret_cast<const float4 *>(v_s + (k + kk) * LDV + j * 64u + tx * 4u);
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        const float w = kk == 0 ? pv[i].x : kk == 1 ? pv[i].y : kk == 2 ? pv[i].z : pv[i].w;
                        o[i][j * 4] = fmaf(w, vv.x, o[i][j * 4]); o[i][j * 4 + 1] = fmaf(w, vv.y, o[i][j * 4 + 1]);
                        o[i][j * 4 + 2] = fmaf(w, vv.z, o[i][j * 4 + 2]); o[i][j * 4 + 3] = fmaf(w, vv.w, o[i][j * 4 + 3]);
                    }
                }
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t rr = r0 + ty * 4u + i;
        if (rr >= rows) continue;
        const uint32_t t = rr / rep, h = g * rep + rr % rep;
        float f = 1.0f / l[i];
        if (a.has_gate) f *= sigmoidf_(a.p[(size_t)t * a.ld + a.g0 + h]);
        float *dst = a.out + ((size_t)t * a.H + h) * VD;
#pragma unroll
        for (int j = 0; j < VJ; j++)
#pragma unroll
            for (int c = 0; c < 4; c++) { const uint32_t n = j * 64u + tx * 4u + c; if (n < VD) dst[n] = o[i][j * 4 + c] * f; }
    }
}

// Short portions (T <= kGemvMaxM): one launch from the joint product's rows to the gated heads.  A block takes one token, hb query heads of
// one key/value head and a share of the key pages.  It norms and turns its own queries (and, where its share reaches the portion's
// tokens, their keys: no block reads a cache row that another block of this launch writes), loads a page's keys and values with every
// load in flight at once (8 lanes per key), and leaves partial (o, m, l) triples; the block that draws the last ticket merges them.
// The block that owns a token's last page also writes the token's cache row.  grid = (key splits, G x head groups, T); 256 threads.
constexpr uint32_t kGqaSplitMax = 64, kGqaHeads = 8;
__host__ __device__ inline uint32_t gqa_vwords(uint32_t VD) { const uint32_t v = kPage * ((VD + 3u) & ~3u), w = kGqaHeads * kGqaSplitMax; return v > w ? v : w; }
inline size_t gqa_decode_smem(uint32_t D, uint32_t VD) { const uint32_t Dp = (D + 3u) & ~3u; return ((size_t)(kGqaHeads + kGemvMaxM) * Dp + gqa_vwords(VD) + 2u * kGqaHeads * kPage) * 4; }
template <int CH, bool VEC>
__global__ void __launch_bounds__(256) k_gqa_decode(const GqaArgs a) {
    pdl_enter();
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[5][8], corr_s[kGqaHeads], l_s[kGqaHeads];
    __shared__ uint32_t last_s;
    const uint32_t D = a.D, VD = a.VD, Dp = (D + 3u) & ~3u, VDp = (VD + 3u) & ~3u, rep = a.H / a.G, hgs = (rep + a.hb - 1u) / a.hb;
    const uint32_t g = blockIdx.y / hgs, h0 = g * rep + (blockIdx.y % hgs) * a.hb, nh = min(a.hb, (g + 1u) * rep - h0), t = blockIdx.z;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, key = tid >> 3, sub = tid & 7u;
    const uint32_t pos = a.pos0 + (a.pos_ptr ? *a.pos_ptr : 0u), nkeys = pos + t + 1u, low = gqa_first(pos + t, a.block), page0 = low / kPage, tiles = (nkeys + kPage - 1u) / kPage - page0;
    const uint32_t tps = (tiles + a.nsplit - 1u) / a.nsplit, nact = (tiles + tps - 1u) / tps, split = blockIdx.x;
    if (split >= nact) return;
    const uint32_t tile_lo = page0 + split * tps, tile_hi = min(page0 + tiles, tile_lo + tps), half = a.tab ? a.half : 0u;
    float *q_s = sm;                                   // [kGqaHeads][Dp]
    float *kn_s = q_s + kGqaHeads * Dp;                // [kGemvMaxM][Dp]: the portion's own keys
    float *v_s = kn_s + kGemvMaxM * Dp;                // [kPage][VDp]
    float *s_s = v_s + gqa_vwords(VD), *p_s = s_s + kGqaHeads * kPage;
    const bool tail = tile_hi * kPage > pos;           // this share holds keys of the portion itself
    const uint32_t V4 = VDp / 4u;
    float4 kr[CH], vr[CH];
    auto fetch = [&](uint32_t tile) {                  // the page's rows of this key/value head; the portion's own tokens come from elsewhere
        const float *pg = a.cache + (size_t)a.table[tile] * kPage * a.RL;
        const uint32_t base = tile * kPage;
        const float *krow = pg + (size_t)key * a.RL + g * D;
#pragma unroll
        for (int c = 0; c < CH; c++) {
            const uint32_t d = (sub + 8u * c) * 4u;
            kr[c] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (base + key < pos && d < Dp) {
                if (VEC) kr[c] = *reinterpret_cast<const float4 *>(krow + d);
                else { kr[c].x = krow[d]; if (d + 1u < D) kr[c].y = krow[d + 1u]; if (d + 2u < D) kr[c].z = krow[d + 2u]; if (d + 3u < D) kr[c].w = krow[d + 3u]; }
            }
        }
#pragma unroll
        for (int c = 0; c < CH; c++) {
            const uint32_t i = tid + 256u * c, k = i / V4, d = (i % V4) * 4u;
            vr[c] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (k >= kPage || base + k >= nkeys) continue;
            const float *src = base + k < pos ? pg + (size_t)k * a.RL + a.G * D + g * VD + d : a.p + (size_t)(base + k - pos) * a.ld + a.v0 + g * VD + d;
            if (VEC) vr[c] = *reinterpret_cast<const float4 *>(src);
            else { vr[c].x = src[0]; if (d + 1u < VD) vr[c].y = src[1]; if (d + 2u < VD) vr[c].z = src[2]; if (d + 3u < VD) vr[c].w = src[3]; }
        }
    };
    fetch(tile_lo);
    // Norm factors are numbers per token: queries and keys are gained and turned without them (no wait for the sums), the scores and the
    // cached key carry them.  red[0]: the whole query row's sum of squares; red[1 + u]: the key row's of the portion's token u (tail shares).
    // Norms per head: red[0][h] is head h's own sum, and one warp makes the whole of red[1 + u].
    const uint32_t QW = a.H * D, KW = a.G * D;
    {
        float s[1 + kGemvMaxM];
#pragma unroll
        for (uint32_t u = 0; u <= kGemvMaxM; u++) s[u] = 0.0f;
        if (a.head_norm) {
            if (a.wq && warp < nh) { const float *q = a.p + (size_t)t * a.ld + a.q0 + (h0 + warp) * D; for (uint32_t i = lane; i < D; i += 32u) s[0] = fmaf(q[i], q[i], s[0]); }
#pragma unroll
            for (uint32_t u = 0; u < kGemvMaxM; u++)
                if (a.wk && tail && u == warp && u <= t) { const float *k = a.p + (size_t)u * a.ld + a.k0 + g * D; for (uint32_t i = lane; i < D; i += 32u) s[1 + u] = fmaf(k[i], k[i], s[1 + u]); }
        } else if (a.wq) {
            const float *q = a.p + (size_t)t * a.ld + a.q0;
            if (VEC) {
#pragma unroll 4
                for (uint32_t i = tid; i < QW / 4u; i += 256u) { const float4 v = reinterpret_cast<const float4 *>(q)[i]; s[0] = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s[0])))); }
            } else for (uint32_t i = tid; i < QW; i += 256u) s[0] = fmaf(q[i], q[i], s[0]);
        }
        if (a.wk && tail && !a.head_norm) {
#pragma unroll
            for (uint32_t u = 0; u < kGemvMaxM; u++)
                if (u <= t) { const float *k = a.p + (size_t)u * a.ld + a.k0; for (uint32_t i = tid; i < KW; i += 256u) s[1 + u] = fmaf(k[i], k[i], s[1 + u]); }
        }
        for (uint32_t i = tid; i < nh * Dp; i += 256u) {
            const uint32_t h = i / Dp, d = i % Dp;
            q_s[i] = d < D ? rot_half_at(a.p + (size_t)t * a.ld + a.q0 + (h0 + h) * D, a.wq ? a.wq + (a.head_norm ? 0u : (h0 + h) * D) : nullptr, 1.0f, d, half, a.tab + (size_t)(pos + t) * half) : 0.0f;
        }
        if (tail)
            for (uint32_t i = tid; i < (t + 1u) * Dp; i += 256u) {
                const uint32_t u = i / Dp, d = i % Dp;
                kn_s[i] = d < D ? rot_half_at(a.p + (size_t)u * a.ld + a.k0 + g * D, a.wk ? a.wk + (a.head_norm ? 0u : g * D) : nullptr, 1.0f, d, half, a.tab + (size_t)(pos + u) * half) : 0.0f;
            }
#pragma unroll
        for (uint32_t u = 0; u <= kGemvMaxM; u++) { s[u] = warp_sum(s[u]); if (lane == 0) red[u][warp] = s[u]; }
    }
    __syncthreads();
    auto factor = [&](uint32_t j, bool normed, uint32_t n) {      // 1 / root mean square of row j of red
        if (!normed) return 1.0f;
        float v = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < 8u; w++) v += red[j][w];
        return 1.0f / sqrtf(v / (float)n + a.eps);
    };
    const uint32_t QN = a.head_norm ? D : QW, KN = a.head_norm ? D : KW;
    const float qf = (a.head_norm && a.wq ? 1.0f / sqrtf(red[0][sub] / (float)QN + a.eps) : factor(0, a.wq != nullptr, QN)) * a.scale;      // of head `sub`, or of all
    if (split == nact - 1u && blockIdx.y % hgs == 0) {            // one block writes the token's row of this key/value head
        float *row = a.cache + ((size_t)a.table[(pos + t) / kPage] * kPage + (pos + t) % kPage) * a.RL;
        const float kf = factor(1u + t, a.wk != nullptr, KN);
        for (uint32_t d = tid; d < D; d += 256u) row[g * D + d] = kn_s[t * Dp + d] * kf;
        for (uint32_t d = tid; d < VD; d += 256u) row[a.G * D + g * VD + d] = a.p[(size_t)t * a.ld + a.v0 + g * VD + d];
    }
    float o[CH], m = -INFINITY, l = 0.0f;              // o: items (head, column) tid, tid + 256, ...; m, l: of head `warp`
#pragma unroll
    for (int c = 0; c < CH; c++) o[c] = 0.0f;
    for (uint32_t tile = tile_lo; tile < tile_hi; tile++) {
        const uint32_t kp = tile * kPage + key;
        if (kp >= pos && kp < nkeys) {
            const float kf = factor(1u + kp - pos, a.wk != nullptr, KN);
#pragma unroll
            for (int c = 0; c < CH; c++) {
                const uint32_t d = (sub + 8u * c) * 4u;
                if (d < Dp) { const float4 v = *reinterpret_cast<const float4 *>(kn_s + (kp - pos) * Dp + d); kr[c] = make_float4(v.x * kf, v.y * kf, v.z * kf, v.w * kf); }
            }
        }
        float acc[kGqaHeads];
#pragma unroll
        for (uint32_t h = 0; h < kGqaHeads; h++) {
            acc[h] = 0.0f;
            if (h < nh) {
#pragma unroll
                for (int c = 0; c < CH; c++) {
                    const uint32_t d = (sub + 8u * c) * 4u;
                    if (d < Dp) { const float4 qv = *reinterpret_cast<const float4 *>(q_s + h * Dp + d); acc[h] = fmaf(qv.w, kr[c].w, fmaf(qv.z, kr[c].z, fmaf(qv.y, kr[c].y, fmaf(qv.x, kr[c].x, acc[h])))); }
                }
            }
        }
#pragma unroll
        for (uint32_t h = 0; h < kGqaHeads; h++) {
            if (h < nh) {
                acc[h] += __shfl_xor_sync(0xffffffffu, acc[h], 4); acc[h] += __shfl_xor_sync(0xffffffffu, acc[h], 2); acc[h] += __shfl_xor_sync(0xffffffffu, acc[h], 1);
                if (sub == h) s_s[h * kPage + key] = acc[h] * qf;
            }
        }
#pragma unroll
        for (int c = 0; c < CH; c++) { const uint32_t i = tid + 256u * c, k = i / V4; if (k < kPage) *reinterpret_cast<float4 *>(v_s + k * VDp + (i % V4) * 4u) = vr[c]; }
        __syncthreads();
        if (warp < nh) {
            float s = s_s[warp * kPage + lane];
            if (a.softcap > 0.0f) s = a.softcap * tanhf(s / a.softcap);
            const bool seen = tile * kPage + lane < nkeys && tile * kPage + lane >= low;
            s = seen ? s : -INFINITY;
            float tm = s;
#pragma unroll
            for (int off = 16; off > 0; off >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, off));
            const float mn = fmaxf(m, tm), corr = expf(m - mn);      // a share's pages all hold a key in sight: mn is finite
            const float pv = seen ? expf(s - mn) : 0.0f;
            l = fmaf(l, corr, warp_sum(pv)); m = mn;
            p_s[warp * kPage + lane] = pv;
            if (lane == 0) corr_s[warp] = corr;
        }
        __syncthreads();
        if (tile + 1u < tile_hi) fetch(tile + 1u);
#pragma unroll
        for (int c = 0; c < CH; c++) {
            const uint32_t i = tid + 256u * c, h = i / VD, d = i % VD;
            if (h < nh) {
                float v = o[c] * corr_s[h];
#pragma unroll
                for (uint32_t k = 0; k < kPage; k += 4u) {
                    const float4 pv = *reinterpret_cast<const float4 *>(p_s + h * kPage + k);
                    v = fmaf(pv.x, v_s[k * VDp + d], v); v = fmaf(pv.y, v_s[(k + 1u) * VDp + d], v);
                    v = fmaf(pv.z, v_s[(k + 2u) * VDp + d], v); v = fmaf(pv.w, v_s[(k + 3u) * VDp + d], v);
                }
                o[c] = v;
            }
        }
        __syncthreads();
    }
    const float *gate = a.p + (size_t)t * a.ld + a.g0;
    if (nact == 1u) {
        if (warp < nh && lane == 0) {
            float den = l, ow = 1.0f;
            if (a.sink) { const float sk = a.sink[h0 + warp], M = fmaxf(m, sk); ow = expf(m - M); den = fmaf(l, ow, expf(sk - M)); }
            l_s[warp] = ow / den * (a.has_gate ? sigmoidf_(gate[h0 + warp]) : 1.0f);
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < CH; c++) { const uint32_t i = tid + 256u * c, h = i / VD; if (h < nh) a.out[((size_t)t * a.H + h0 + h) * VD + i % VD] = o[c] * l_s[h]; }
        return;
    }
    // partial triples, then the last block of this (token, head group) merges:
    //   out = gate sum_s e^{m_s - M} o_s / (sum_s e^{m_s - M} l_s + e^{sink - M})
    const uint32_t PW = VD + 2u;
    float *mine = a.part + (((size_t)t * kGqaSplitMax + split) * a.H + h0) * PW;
#pragma unroll
    for (int c = 0; c < CH; c++) { const uint32_t i = tid + 256u * c, h = i / VD; if (h < nh) mine[h * PW + i % VD] = o[c]; }
    if (warp < nh && lane == 0) { mine[warp * PW + VD] = m; mine[warp * PW + VD + 1u] = l; }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        uint32_t *tk = a.tickets + blockIdx.z * gridDim.y + blockIdx.y;
        const uint32_t got = atomicAdd(tk, 1u);
        last_s = got + 1u == nact;
        if (last_s) *tk = 0u;              // ready for the next launch
    }
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    const size_t stride = (size_t)a.H * PW;
    const float *base = a.part + ((size_t)t * kGqaSplitMax * a.H + h0) * PW;
    float *w_s = v_s;                      // [kGqaHeads][kGqaSplitMax]
    if (warp < nh) {
        float ms[2], ls[2], M = a.sink ? a.sink[h0 + warp] : -INFINITY;
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const uint32_t sp = lane + 32u * k;
            ms[k] = sp < nact ? __ldcg(base + sp * stride + warp * PW + VD) : -INFINITY;
            ls[k] = sp < nact ? __ldcg(base + sp * stride + warp * PW + VD + 1u) : 0.0f;
            M = fmaxf(M, ms[k]);
        }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, off));
        float L = 0.0f;
#pragma unroll
        for (int k = 0; k < 2; k++) { ms[k] = expf(ms[k] - M); L = fmaf(ms[k], ls[k], L); }
        L = warp_sum(L);
        if (a.sink) L += expf(a.sink[h0 + warp] - M);
        const float f = (a.has_gate ? sigmoidf_(gate[h0 + warp]) : 1.0f) / L;
#pragma unroll
        for (int k = 0; k < 2; k++) w_s[warp * kGqaSplitMax + lane + 32u * k] = ms[k] * f;
    }
    __syncthreads();
    float acc[CH];
    const float *src[CH]; const float *wr[CH]; bool ok[CH];
#pragma unroll
    for (int c = 0; c < CH; c++) {
        const uint32_t i = tid + 256u * c, h = i / VD;
        ok[c] = h < nh; acc[c] = 0.0f;
        src[c] = base + (ok[c] ? h * PW + i % VD : 0u); wr[c] = w_s + (ok[c] ? h : 0u) * kGqaSplitMax;
    }
#pragma unroll 8
    for (uint32_t sp = 0; sp < nact; sp++)
#pragma unroll
        for (int c = 0; c < CH; c++) if (ok[c]) acc[c] = fmaf(wr[c][sp], __ldcg(src[c] + sp * stride), acc[c]);
#pragma unroll
    for (int c = 0; c < CH; c++) { const uint32_t i = tid + 256u * c; if (ok[c]) a.out[((size_t)t * a.H + h0 + i / VD) * VD + i % VD] = acc[c]; }
}

// ------------------------------------------------------------------------------------------------
// Gated delta rule.  Channels [q G D | k G D | v H VD] of the joint product pass a causal convolution (taps [C][K], tail [K - 1][C] in
// the state, no bias) and silu; head h uses q/k head h / (H / G).  State [H][VD][D] fp32: column j of head h is contiguous.
//
// Long portions solve kDeltaChunk tokens together.  With Gm_i = g_1 .. g_i (products inside the chunk, per channel) and S the state
// before it, the recurrence gives
//     p_i = S^T (Gm_i k_i) + sum_{j<i} A_ij u_j,    A_ij = sum_d k_i k_j prod_{j<l<=i} g_l,    u_i = beta_i (v_i - p_i)
//     o_i = S^T (Gm_i q_i) + sum_{j<=i} B_ij u_j,   B_ij = sum_d q_i k_j prod_{j<l<=i} g_l
//     S  <- Gm_C S + sum_j (prod_{l>j} g_l k_j) u_j^T
// so  u = M_u w  and  o = S^T (Gm q) + M_o w  with  w_j = v_j - S^T (Gm_j k_j)  and two 4 x 4 triangular matrices made of A, B and beta alone:
// a value column meets its state twice per chunk instead of twice per token, and the sums over the key coordinates of all its
// tokens run side by side.  Every product of decays is a product of numbers in (0, 1], never a quotient.
// ------------------------------------------------------------------------------------------------
constexpr uint32_t kDeltaChunk = 4, kDeltaDim = 256, kDeltaVecs = 3 * kDeltaChunk + 1, kDeltaMat = 2 * kDeltaChunk * kDeltaChunk;
// what the scan reads of a chunk and head, in one run: Gm_i k_i (4), Gm_i q_i (4), prod_{l>j} g_l k_j (4), Gm_C, each `dp` coordinates; M_u, M_o
__host__ __device__ inline uint32_t delta_dp(uint32_t D) { return D <= 32u ? 32u : D <= 64u ? 64u : D <= 128u ? 128u : 256u; }
__host__ __device__ inline uint32_t delta_block(uint32_t dp) { return kDeltaVecs * dp + kDeltaMat; }
// exp(-rate sp), in double precision and rounded once: a state that forgets slowly takes thousands of these factors
__device__ __forceinline__ float delta_decay(float rate, float sp) { return (float)exp(-(double)rate * (double)sp); }

struct DeltaPrepArgs {
    const float *p; uint32_t ld, c0, b0, a0; const float *taps; const float *state; uint32_t K;      // c0: the first convolved channel's column
    const float *sp;                       // per-channel decay: softplus already taken, [T][H D]; null: one decay per head from column a0 + h
    const float *dt_bias, *rate;
    float *blk, *v;                        // blk [chunks][H][delta_block], v [T][H VD]
    uint32_t T, H, G, D, VD; float qscale;
};
// grid = (chunks, heads), delta_dp(D) threads: a thread makes the chunk's tokens of its key coordinate (and of some value columns).  All sums
// over the coordinates -- squares, and the products between tokens -- are taken of the vectors before they become unit vectors, in one
// reduction; their factors join afterwards.
__global__ void __launch_bounds__(kDeltaDim) k_delta_prep(const DeltaPrepArgs a) {
    pdl_enter();
    constexpr uint32_t C4 = kDeltaChunk;
    __shared__ float red[8][32], tot[32], fac[2 * C4], beta_s[C4];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, nw = blockDim.x >> 5, DP = blockDim.x, t0 = blockIdx.x * C4, h = blockIdx.y, g = h / (a.H / a.G);
    const uint32_t D = a.D, GD = a.G * D, C = 2u * GD + a.H * a.VD, K = a.K;
    float *blk = a.blk + ((size_t)blockIdx.x * a.H + h) * delta_block(DP);
    // one row of channel c before (or in) the portion
    auto input = [&](int32_t src, uint32_t c) {
        return src >= 0 ? (src < (int32_t)a.T ? a.p[(size_t)src * a.ld + a.c0 + c] : 0.0f) : a.state[(size_t)((int32_t)(K - 1u) + src) * C + c];
    };
    float q[C4], k[C4], gv[C4];
#pragma unroll
    for (uint32_t i = 0; i < C4; i++) { q[i] = 0.0f; k[i] = 0.0f; gv[i] = 1.0f; }
    const float rate = a.rate[h];
    if (tid < D) {
        const uint32_t cq = g * D + tid, ck = GD + cq;
        float wq[C4], wk[C4];              // the taps that meet input m for tokens 0..3: taps[m - i]
#pragma unroll
        for (uint32_t i = 0; i < C4; i++) { wq[i] = 0.0f; wk[i] = 0.0f; }
#pragma unroll 4
        for (uint32_t m = 0; m < K + C4 - 1u; m++) {
            const int32_t src = (int32_t)(t0 + m) - (int32_t)(K - 1u);
            const float xq = input(src, cq), xk = input(src, ck);
#pragma unroll
            for (int i = (int)C4 - 1; i > 0; i--) { wq[i] = wq[i - 1]; wk[i] = wk[i - 1]; }
            wq[0] = m < K ? a.taps[(size_t)cq * K + m] : 0.0f; wk[0] = m < K ? a.taps[(size_t)ck * K + m] : 0.0f;
#pragma unroll
            for (uint32_t i = 0; i < C4; i++) { q[i] = fmaf(wq[i], xq, q[i]); k[i] = fmaf(wk[i], xk, k[i]); }
        }
#pragma unroll
        for (uint32_t i = 0; i < C4; i++) {
            const uint32_t t = t0 + i;
            if (t < a.T) {
                q[i] = siluf_(q[i]); k[i] = siluf_(k[i]);
                gv[i] = delta_decay(rate, a.sp ? a.sp[((size_t)t * a.H + h) * D + tid] : softplusf_(a.p[(size_t)t * a.ld + a.a0 + h] + a.dt_bias[h]));
            } else { q[i] = 0.0f; k[i] = 0.0f; }      // tokens past the portion: nothing is forgotten, nothing is written
        }
    }
    if (tid < C4) beta_s[tid] = t0 + tid < a.T ? sigmoidf_(a.p[(size_t)(t0 + tid) * a.ld + a.b0 + h]) : 0.0f;
    // sums 0..3: q_i^2, 4..7: k_i^2, 8 + i (i - 1) / 2 + j: k_i k_j prod_{j<l<=i} g_l (j < i), 14 + i (i + 1) / 2 + j: q_i k_j prod (j <= i)
    float x[32];
#pragma unroll
    for (int i = 0; i < 32; i++) x[i] = 0.0f;
#pragma unroll
    for (int i = 0; i < (int)C4; i++) {
        x[i] = q[i] * q[i]; x[4 + i] = k[i] * k[i];
        float dec = 1.0f;
#pragma unroll
        for (int j = i; j >= 0; j--) {
            if (j < i) { dec *= gv[j + 1]; x[8 + i * (i - 1) / 2 + j] = k[i] * k[j] * dec; }
            x[14 + i * (i + 1) / 2 + j] = q[i] * k[j] * dec;
        }
    }
    // 32 sums over 32 lanes: lane l ends with sum l
#pragma unroll
    for (int half = 16; half > 0; half >>= 1) {
        const bool up = lane & half;
#pragma unroll
        for (int i = 0; i < half; i++) {
            const float keep = up ? x[i + half] : x[i], give = up ? x[i] : x[i + half];
            x[i] = keep + __shfl_xor_sync(0xffffffffu, give, half);
        }
    }
    red[warp][lane] = x[0];
    // the value columns, meanwhile
    for (uint32_t j = tid; j < a.VD; j += blockDim.x) {
        const uint32_t cv = 2u * GD + h * a.VD + j;
        float v[C4], wv[C4];
#pragma unroll
        for (uint32_t i = 0; i < C4; i++) { v[i] = 0.0f; wv[i] = 0.0f; }
#pragma unroll 4
        for (uint32_t m = 0; m < K + C4 - 1u; m++) {
            const float xv = input((int32_t)(t0 + m) - (int32_t)(K - 1u), cv);
#pragma unroll
            for (int i = (int)C4 - 1; i > 0; i--) wv[i] = wv[i - 1];
            wv[0] = m < K ? a.taps[(size_t)cv * K + m] : 0.0f;
#pragma unroll
            for (uint32_t i = 0; i < C4; i++) v[i] = fmaf(wv[i], xv, v[i]);
        }
#pragma unroll
        for (uint32_t i = 0; i < C4; i++) if (t0 + i < a.T) a.v[(size_t)(t0 + i) * a.H * a.VD + h * a.VD + j] = siluf_(v[i]);
    }
    __syncthreads();
    if (tid < 32u) {
        float s = 0.0f;
        for (uint32_t w = 0; w < nw; w++) s += red[w][tid];
        tot[tid] = s;
        if (tid < 2u * C4) fac[tid] = (tid < C4 ? a.qscale : 1.0f) / sqrtf(s + 1e-6f);      // the unit vectors' factors: q 0..3, k 4..7
    }
    __syncthreads();
    {
        float pre = 1.0f, suf = 1.0f;
#pragma unroll
        for (uint32_t i = 0; i < C4; i++) {
            pre *= gv[i];
            k[i] *= fac[C4 + i];
            blk[i * DP + tid] = pre * k[i];
            blk[(C4 + i) * DP + tid] = pre * (q[i] * fac[i]);
        }
#pragma unroll
        for (int i = (int)C4 - 1; i >= 0; i--) { blk[(2u * C4 + i) * DP + tid] = suf * k[i]; suf *= gv[i]; }
        blk[3u * C4 * DP + tid] = pre;
    }
    // w = v - S^T (Gm k)  ->  u = M_u w with rows M_i = beta_i (e_i - sum_{j<i} A_ij M_j), and o = S^T (Gm q) + (B M_u) w: column `tid` of both
    if (tid < C4) {
        float M[C4], *mat = blk + kDeltaVecs * DP;
#pragma unroll
        for (int i = 0; i < (int)C4; i++) {
            float v = i == (int)tid ? 1.0f : 0.0f;
#pragma unroll
            for (int j = 0; j < i; j++) v = fmaf(-tot[8 + i * (i - 1) / 2 + j] * fac[C4 + i] * fac[C4 + j], M[j], v);
            M[i] = beta_s[i] * v;
            mat[i * C4 + tid] = M[i];
        }
#pragma unroll
        for (int i = 0; i < (int)C4; i++) {
            float v = 0.0f;
#pragma unroll
            for (int j = 0; j <= i; j++) v = fmaf(tot[14 + i * (i + 1) / 2 + j] * fac[i] * fac[C4 + j], M[j], v);
            mat[C4 * C4 + i * C4 + tid] = v;
        }
    }
}

// A block of 8 warps owns 16 value columns of head h = blockIdx.y, a warp two of them; the 32 lanes share the key coordinates.  A chunk
// takes 8 sums over the coordinates per column (four S^T (Gm_i k_i), four S^T (Gm_i q_i)); the warp reduces its 16 sums with 16 shuffles
// and no selection, because lane l keeps sum (i, column c) in the place (i ^ (l / 4), c ^ (l / 2 % 2)) from the start -- it reads the chunk
// vectors in that order and its two columns of the state sit in that order.  Lanes 2 n and 2 n + 1 end with sum n.  Tiles of NCH chunks
// travel two ahead (cp.async into a ring of three).
struct DeltaScanArgs { const float *blk, *v; float *S; float *o; uint32_t T, H, D, VD; };
template <int VW> __device__ __forceinline__ void lds_vec(const float *p, float *v) {
    if constexpr (VW == 4) { const float4 f = *reinterpret_cast<const float4 *>(p); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
    else if constexpr (VW == 2) { const float2 f = *reinterpret_cast<const float2 *>(p); v[0] = f.x; v[1] = f.y; }
    else v[0] = *p;
}
__device__ __forceinline__ void cp_async4(float *dst, const float *src, bool ok) {      // 4 bytes into shared memory; zero when !ok
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst), n = ok ? 4u : 0u;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
template <int DCH>
__global__ void __launch_bounds__(256, 2) k_delta_scan(const DeltaScanArgs a) {
    pdl_enter();
    constexpr uint32_t DP = DCH * 32u, NCH = DCH <= 4 ? 2u : 1u, BLK = kDeltaVecs * DP + kDeltaMat;
    constexpr int VW = DCH < 4 ? DCH : 4, NB = DCH / VW;      // a lane's coordinates: NB runs of VW, at (run * 32 + lane) * VW
    __shared__ __align__(16) float w_s[3][NCH][BLK];
    __shared__ __align__(16) float v_s[3][NCH][4][16];
    __shared__ __align__(16) float u_s[8][2][2][4];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, li = lane >> 2, lc = (lane >> 1) & 1u, h = blockIdx.y, col0 = blockIdx.x * 16u, jw = col0 + warp * 2u;
    const uint32_t D = a.D, HV = a.H * a.VD, chunks = (a.T + kDeltaChunk - 1u) / kDeltaChunk, tiles = (chunks + NCH - 1u) / NCH;
    auto fetch = [&](uint32_t tile) {          // one group of copies per tile, an empty one past the last
        if (tile < tiles) {
            const uint32_t st = tile % 3u, ch0 = tile * NCH;
            for (uint32_t i = tid; i < NCH * (BLK / 4u); i += 256u) {
                const uint32_t c = i / (BLK / 4u), e = (i % (BLK / 4u)) * 4u;
                if (ch0 + c < chunks) cp_async16(&w_s[st][c][e], a.blk + ((size_t)(ch0 + c) * a.H + h) * BLK + e, true);
            }
            if (tid < NCH * 64u) {
                const uint32_t c = tid / 64u, i = (tid / 16u) % 4u, j = tid % 16u, t = (ch0 + c) * kDeltaChunk + i;
                const bool ok = t < a.T && col0 + j < a.VD;
                cp_async4(&v_s[st][c][i][j], ok ? a.v + (size_t)t * HV + h * a.VD + col0 + j : a.v, ok);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0); fetch(1);
    float S[2][DCH];                           // S[c]: column jw + (c ^ lc)
#pragma unroll
    for (uint32_t c = 0; c < 2; c++)
#pragma unroll
        for (int e = 0; e < DCH; e++) {
            const uint32_t d = ((e / VW) * 32u + lane) * VW + e % VW, col = jw + (c ^ lc);
            S[c][e] = (col < a.VD && d < D) ? a.S[((size_t)h * a.VD + col) * D + d] : 0.0f;
        }
    for (uint32_t tile = 0; tile < tiles; tile++) {
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();                       // this tile has landed for every thread, and the one before is done with: its place is free
        fetch(tile + 2u);
        const uint32_t st = tile % 3u;
#pragma unroll
        for (uint32_t c = 0; c < NCH; c++) {
            if (tile * NCH + c >= chunks) break;
            const float *w = &w_s[st][c][lane * VW], *mat = &w_s[st][c][kDeltaVecs * DP];
            float x[8][2];
#pragma unroll
            for (uint32_t i = 0; i < 8; i++) {
                float f[DCH];
#pragma unroll
                for (int n = 0; n < NB; n++) lds_vec<VW>(w + (i ^ li) * DP + n * 32 * VW, f + n * VW);
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    x[i][j] = S[j][0] * f[0];
#pragma unroll
                    for (int e = 1; e < DCH; e++) x[i][j] = fmaf(S[j][e], f[e], x[i][j]);
                }
            }
#pragma unroll
            for (int half = 4; half > 0; half >>= 1)
#pragma unroll
                for (int i = 0; i < half; i++)
#pragma unroll
                    for (int j = 0; j < 2; j++) x[i][j] += __shfl_xor_sync(0xffffffffu, x[i + half][j], half * 4);
            float mine = x[0][0] + __shfl_xor_sync(0xffffffffu, x[0][1], 2);
            mine += __shfl_xor_sync(0xffffffffu, mine, 1);      // lanes 0..15: S^T (Gm_i k_i), 16..31: S^T (Gm_i q_i), i = li % 4, column jw + lc
            const float wj = v_s[st][c][li & 3u][warp * 2u + lc] - mine;
            const float4 mr = *reinterpret_cast<const float4 *>(mat + li * 4u);
            float y = li < 4u ? 0.0f : mine;
            y = fmaf(mr.x, __shfl_sync(0xffffffffu, wj, lc * 2u), y); y = fmaf(mr.y, __shfl_sync(0xffffffffu, wj, 4u + lc * 2u), y);
            y = fmaf(mr.z, __shfl_sync(0xffffffffu, wj, 8u + lc * 2u), y); y = fmaf(mr.w, __shfl_sync(0xffffffffu, wj, 12u + lc * 2u), y);
            if ((lane & 1u) == 0) {
                if (li < 4u) u_s[warp][c & 1u][lc][li] = y;
                else {
                    const uint32_t t = (tile * NCH + c) * kDeltaChunk + (li & 3u);
                    if (t < a.T && jw + lc < a.VD) a.o[(size_t)t * HV + h * a.VD + jw + lc] = y;
                }
            }
            float f[5][DCH];                   // the writes' keys, decayed to the chunk's end, and the chunk's whole decay
#pragma unroll
            for (int i = 0; i < 5; i++)
#pragma unroll
                for (int n = 0; n < NB; n++) lds_vec<VW>(w + (8 + i) * DP + n * 32 * VW, f[i] + n * VW);
            __syncwarp();
            float u[2][4];                     // u[c]: the four tokens' steps of column jw + (c ^ lc)
#pragma unroll
            for (uint32_t j = 0; j < 2; j++) lds_vec<4>(&u_s[warp][c & 1u][j ^ lc][0], u[j]);
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int e = 0; e < DCH; e++) {
                    float v = S[j][e] * f[4][e];
#pragma unroll
                    for (int i = 0; i < 4; i++) v = fmaf(f[i][e], u[j][i], v);
                    S[j][e] = v;
                }
        }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
#pragma unroll
    for (uint32_t c = 0; c < 2; c++)
#pragma unroll
        for (int e = 0; e < DCH; e++) {
            const uint32_t d = ((e / VW) * 32u + lane) * VW + e % VW, col = jw + (c ^ lc);
            if (col < a.VD && d < D) a.S[((size_t)h * a.VD + col) * D + d] = S[c][e];
        }
}

// Short portions (T <= kGemvMaxM): a cluster of blocks per head, each with a share of its value columns, from the convolved channels (an
// epilogue of the joint product) to the normed and gated output; the blocks exchange their parts of the decays and their columns' sums of
// squares through each other's shared memory.  8 lanes share a value column.  Low-rank decay and gate: their second products, W_a2 (a1) and W_g2 (g1) with a1, g1
// columns of the joint product, are made here for the head's own rows (round_a: the operand rounded to bf16 first, as a tensor-core
// product would).  Without them the decay is one number per head (column a0 + h) and the gate silu of H VD columns at g0.
constexpr uint32_t kDeltaBlocks = 4;       // blocks per head at most
__host__ __device__ inline uint32_t delta_step_blocks(uint32_t VD) { return VD >= 64u ? 4u : VD >= 32u ? 2u : 1u; }
__host__ __device__ inline uint32_t delta_step_cols(uint32_t VD) { const uint32_t n = delta_step_blocks(VD); return ((VD + n - 1u) / n + 3u) & ~3u; }
struct DeltaStepArgs {
    const float *cv; const float *p; uint32_t ld, b0, a0, g0; const void *a2, *g2; uint32_t ra, rg; const float *dt_bias, *rate, *gain;
    float *S; float *out; uint32_t T, H, G, D, VD; float qscale, eps; uint32_t round_a;
};
inline size_t delta_step_smem(int dch, uint32_t VD) { return ((size_t)3 * kGemvMaxM * (uint32_t)dch * 32u + (size_t)2 * kGemvMaxM * delta_step_cols(VD)) * 4; }      // dch: the instance's, DCH
// dot products of one weight row with up to kGemvMaxM rows of x (stride ld), 8 lanes per row; every lane gets the totals.  vec: 16-byte
// loads of both operands are aligned
template <typename WT>
__device__ __forceinline__ void lane8_dots(const WT *w, const float *x, uint32_t ld, uint32_t rows, uint32_t n, bool vec, bool rnd, uint32_t sub, float (&acc)[kGemvMaxM]) {
    constexpr uint32_t VN = WVec<WT>::N;
#pragma unroll
    for (uint32_t t = 0; t < kGemvMaxM; t++) acc[t] = 0.0f;
    const uint32_t nv = vec ? n / VN * VN : 0u;
    for (uint32_t e = sub * VN; e < nv; e += 8u * VN) {
        float wv[VN];
        WVec<WT>::load(w + e, wv);
#pragma unroll
        for (uint32_t t = 0; t < kGemvMaxM; t++)
            if (t < rows) {
#pragma unroll
                for (uint32_t j = 0; j < VN; j += 4u) {
                    const float4 v = *reinterpret_cast<const float4 *>(x + (size_t)t * ld + e + j);
                    const float f[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                    for (int q = 0; q < 4; q++) acc[t] = fmaf(wv[j + q], rnd ? round_bf16(f[q]) : f[q], acc[t]);
                }
            }
    }
    for (uint32_t e = nv + sub; e < n; e += 8u) {
        const float wv = wval(w + e);
#pragma unroll
        for (uint32_t t = 0; t < kGemvMaxM; t++) if (t < rows) { const float v = x[(size_t)t * ld + e]; acc[t] = fmaf(wv, rnd ? round_bf16(v) : v, acc[t]); }
    }
#pragma unroll
    for (uint32_t t = 0; t < kGemvMaxM; t++) { acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], 4); acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], 2); acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], 1); }
}
constexpr uint32_t kDeltaThreads = 512;    // a block's threads at most (8 per value column; more columns: several passes)
template <typename WT, int DCH>
__global__ void __launch_bounds__(kDeltaThreads) k_delta_step(const DeltaStepArgs a) {
    pdl_launch_next();
    cluster_arrive();                          // waited for before the first access to another block's shared memory
    constexpr uint32_t DP = DCH * 32u;
    extern __shared__ __align__(16) float sm[];
    __shared__ float kq_s[kGemvMaxM], beta_s[kGemvMaxM], ss_s[kGemvMaxM][kDeltaBlocks];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, sub = lane & 7u, nw = blockDim.x >> 5, h = blockIdx.y, D = a.D, VD = a.VD, T = a.T;
    const uint32_t CB = delta_step_cols(VD), col_lo = min(VD, blockIdx.x * CB), nc = min(VD, col_lo + CB) - col_lo;      // this block's value columns
    const WT *a2 = static_cast<const WT *>(a.a2), *g2 = static_cast<const WT *>(a.g2);
    const uint32_t part = DP / gridDim.x, lo = blockIdx.x * part, hi = lo + part;      // this block's share of the head's decays
    if (a2 && lo < D) prefetch_weight_rows(a2 + ((size_t)h * D + lo) * a.ra, sizeof(WT), a.ra, a.ra, min(hi, D) - lo, warp, nw, 8u);
    if (g2) prefetch_weight_rows(g2 + ((size_t)h * VD + col_lo) * a.rg, sizeof(WT), a.rg, a.rg, nc, warp, nw, 4u);
    pdl_wait();
    float *q_s = sm, *k_s = q_s + kGemvMaxM * DP, *g_s = k_s + kGemvMaxM * DP, *o_s = g_s + kGemvMaxM * DP, *gate_s = o_s + kGemvMaxM * CB;
    const uint32_t GD = a.G * D, C = 2u * GD + a.H * VD, gk = (h / (a.H / a.G)) * D, groups = blockDim.x >> 3;
    const bool dvec = (D & 3u) == 0;
    float S[DCH][4], v_r[kGemvMaxM];
    // a column's state and its values of every token; j: column of this block
    auto load_column = [&](uint32_t j) {
        const float *Sp = a.S + ((size_t)h * VD + col_lo + j) * D;
#pragma unroll
        for (int c = 0; c < DCH; c++) {
            const uint32_t d = (sub + 8u * c) * 4u;
#pragma unroll
            for (int e = 0; e < 4; e++) S[c][e] = 0.0f;
            if (j < nc && d < D) {
                if (dvec) { const float4 v = *reinterpret_cast<const float4 *>(Sp + d); S[c][0] = v.x; S[c][1] = v.y; S[c][2] = v.z; S[c][3] = v.w; }
                else {
#pragma unroll
                    for (uint32_t e = 0; e < 4; e++) if (d + e < D) S[c][e] = Sp[d + e];
                }
            }
        }
#pragma unroll
        for (uint32_t t = 0; t < kGemvMaxM; t++) v_r[t] = (t < T && j < nc) ? a.cv[(size_t)t * C + 2u * GD + h * VD + col_lo + j] : 0.0f;
    };
    load_column(tid >> 3);                     // in flight while the vectors are made
    const float rate = a.rate[h];
    for (uint32_t t = warp; t < T; t += nw) {  // unit vectors of a token
        const float *q = a.cv + (size_t)t * C + gk, *k = q + GD;
        float qr[DCH], kr[DCH], sq = 0.0f, sk = 0.0f, sx = 0.0f;
        const float braw = a.p[(size_t)t * a.ld + a.b0 + h], araw = a2 ? 0.0f : a.p[(size_t)t * a.ld + a.a0 + h] + a.dt_bias[h];
#pragma unroll
        for (int c = 0; c < DCH; c++) { const uint32_t d = lane + 32u * c; qr[c] = d < D ? q[d] : 0.0f; kr[c] = d < D ? k[d] : 0.0f; }
#pragma unroll
        for (int c = 0; c < DCH; c++) { sq = fmaf(qr[c], qr[c], sq); sk = fmaf(kr[c], kr[c], sk); sx = fmaf(qr[c], kr[c], sx); }
        sq = warp_sum(sq); sk = warp_sum(sk); sx = warp_sum(sx);
        const float rq = a.qscale / sqrtf(sq + 1e-6f), rk = 1.0f / sqrtf(sk + 1e-6f), gh = a2 ? 1.0f : delta_decay(rate, softplusf_(araw));
#pragma unroll
        for (int c = 0; c < DCH; c++) { const uint32_t d = t * DP + lane + 32u * c; q_s[d] = qr[c] * rq; k_s[d] = kr[c] * rk; if (!a2) g_s[d] = gh; }
        if (lane == 0) { kq_s[t] = sx * rq * rk; beta_s[t] = sigmoidf_(braw); }
    }
    if (a2) {
        const bool vec = a.ra % WVec<WT>::N == 0 && ((a.a0 | a.ld) & 3u) == 0 && (reinterpret_cast<uintptr_t>(a2) & 15u) == 0;
        // the head's decays are shared work: every block makes its part of the rows and hands them to all blocks of the head
        __syncwarp();
        cluster_wait();                        // every block of the cluster runs
        for (uint32_t r0 = lo; r0 < hi; r0 += groups) {      // a warp's lanes stay together: the row sums are shuffles
            const uint32_t r = r0 + (tid >> 3), rr = h * D + min(r, D - 1u);
            const float bias = a.dt_bias[rr];
            float z[kGemvMaxM];
            lane8_dots<WT>(a2 + (size_t)rr * a.ra, a.p + a.a0, a.ld, T, a.ra, vec, a.round_a != 0, sub, z);
            if (sub < T && r < hi) {
                const float gv = r < D ? delta_decay(rate, softplusf_(pick_row(z, (int32_t)sub) + bias)) : 1.0f;
                for (uint32_t b = 0; b < gridDim.x; b++) st_cluster(&g_s[sub * DP + r], b, gv);
            }
        }
    }
    if (g2) {
        const bool vec = a.rg % WVec<WT>::N == 0 && ((a.g0 | a.ld) & 3u) == 0 && (reinterpret_cast<uintptr_t>(g2) & 15u) == 0;
        for (uint32_t r0 = 0; r0 < nc; r0 += groups) {
            const uint32_t r = r0 + (tid >> 3);
            float z[kGemvMaxM];
            lane8_dots<WT>(g2 + ((size_t)h * VD + col_lo + min(r, nc - 1u)) * a.rg, a.p + a.g0, a.ld, T, a.rg, vec, a.round_a != 0, sub, z);
            if (sub < T && r < nc) gate_s[sub * CB + r] = sigmoidf_(pick_row(z, (int32_t)sub)) * a.gain[col_lo + r];
        }
    } else for (uint32_t i = tid; i < T * nc; i += blockDim.x) gate_s[(i / nc) * CB + i % nc] = siluf_(a.p[(size_t)(i / nc) * a.ld + a.g0 + h * VD + col_lo + i % nc]) * a.gain[col_lo + i % nc];
    __syncwarp();
    if (a2) { cluster_arrive(); cluster_wait(); } else __syncthreads();
    for (uint32_t c0 = 0; c0 < nc; c0 += groups) {
        const uint32_t j = c0 + (tid >> 3);
        if (c0) load_column(j);
#pragma unroll
        for (uint32_t t = 0; t < kGemvMaxM; t++) {
            if (t >= T) break;
            float pk = 0.0f, pq = 0.0f;
#pragma unroll
            for (int c = 0; c < DCH; c++) {
                const uint32_t d = t * DP + (sub + 8u * c) * 4u;
                const float4 gv = *reinterpret_cast<const float4 *>(g_s + d), kv = *reinterpret_cast<const float4 *>(k_s + d), qv = *reinterpret_cast<const float4 *>(q_s + d);
                S[c][0] *= gv.x; S[c][1] *= gv.y; S[c][2] *= gv.z; S[c][3] *= gv.w;
                pk = fmaf(S[c][3], kv.w, fmaf(S[c][2], kv.z, fmaf(S[c][1], kv.y, fmaf(S[c][0], kv.x, pk))));
                pq = fmaf(S[c][3], qv.w, fmaf(S[c][2], qv.z, fmaf(S[c][1], qv.y, fmaf(S[c][0], qv.x, pq))));
            }
#pragma unroll
            for (int off = 4; off > 0; off >>= 1) { pk += __shfl_xor_sync(0xffffffffu, pk, off); pq += __shfl_xor_sync(0xffffffffu, pq, off); }
            const float u = beta_s[t] * (v_r[t] - pk);
            if (sub == 0 && j < nc) o_s[t * CB + j] = fmaf(kq_s[t], u, pq);
#pragma unroll
            for (int c = 0; c < DCH; c++) {
                const float4 kv = *reinterpret_cast<const float4 *>(k_s + t * DP + (sub + 8u * c) * 4u);
                S[c][0] = fmaf(kv.x, u, S[c][0]); S[c][1] = fmaf(kv.y, u, S[c][1]); S[c][2] = fmaf(kv.z, u, S[c][2]); S[c][3] = fmaf(kv.w, u, S[c][3]);
            }
        }
        if (j < nc) {
            float *Sp = a.S + ((size_t)h * VD + col_lo + j) * D;
#pragma unroll
            for (int c = 0; c < DCH; c++) {
                const uint32_t d = (sub + 8u * c) * 4u;
                if (d >= D) continue;
                if (dvec) *reinterpret_cast<float4 *>(Sp + d) = make_float4(S[c][0], S[c][1], S[c][2], S[c][3]);
                else {
#pragma unroll
                    for (uint32_t e = 0; e < 4; e++) if (d + e < D) Sp[d + e] = S[c][e];
                }
            }
        }
    }
    __syncthreads();
    if (!a2) cluster_wait();                   // every block of the cluster runs
    for (uint32_t t = warp; t < T; t += nw) {  // this block's share of the head's sum of squares, to every block of the head
        float s = 0.0f;
        for (uint32_t j = lane; j < nc; j += 32u) s = fmaf(o_s[t * CB + j], o_s[t * CB + j], s);
        s = warp_sum(s);
        if (lane < gridDim.x) st_cluster(&ss_s[t][blockIdx.x], lane, s);
    }
    __syncwarp();
    cluster_arrive();
    cluster_wait();
    for (uint32_t i = tid; i < T * nc; i += blockDim.x) {
        const uint32_t t = i / nc, j = i % nc;
        float s = 0.0f;
        for (uint32_t r = 0; r < gridDim.x; r++) s += ss_s[t][r];
        a.out[((size_t)t * a.H + h) * VD + col_lo + j] = o_s[t * CB + j] / sqrtf(s / (float)VD + a.eps) * gate_s[t * CB + j];
    }
}

}  // namespace lm
}  // namespace nb
