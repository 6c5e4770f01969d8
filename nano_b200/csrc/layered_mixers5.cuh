// layered_mixers5.cuh -- more mechanisms of the layered runtime (layered.cu), under the rules of layered_kernels.cuh: a kernel per
// mechanism, constants as arguments, fp32 (or more) for everything that is not a matrix-product operand.
//
//   norms after the sum  k_post_ln (x = unit(alpha x + sublayer output) w, where the output may be the weighted rows of routed experts)
//   matrix memory        per head  m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T,  n likewise with k alone;
//                        o = S^T q / (max(|n . q|, e^(-m')) + 1e-6),  i, f the logs of the gates, soft-capped.
//                        Long portions run kMemChunk tokens side by side: k_memory_gates (gates, their running sums and the running
//                        maximum), k_memory_writes (what every chunk writes), k_memory_chain (the state before every chunk), k_memory_out
//                        (all outputs of a chunk: a decayed causal product inside it and one product with the state before it).  k_memory_step (short portions): everything from the
//                        joint product's rows to the normed and gated output, a cluster of blocks per head.
#pragma once
#include "layered_mixers4.cuh"

namespace nb {
namespace lm {

// ------------------------------------------------------------------------------------------------
// x[t] = u / rms(u) w  with  u = alpha x[t] + d[t],  or (eo given)  u = alpha x[t] + sum_j wt[t][j] eo[slot[t][j]];  keep (optional)
// receives the updated x.  One block per token.  NV > 0: a thread keeps its (at most NV) runs of VW neighbours in registers across the
// reduction; VW 4: rows are multiples of 4 and travel in 16-byte pieces.
// ------------------------------------------------------------------------------------------------
struct PostLnArgs { float *x; const float *d; const float *eo; const uint32_t *slot; const float *wt; uint32_t top; const float *w; float alpha; float *keep; uint32_t T, E; float eps; };
template <int VW> __device__ __forceinline__ void stg_vec(float *p, const float (&v)[VW]) {
    if constexpr (VW == 4) *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}
template <int NV, int VW>
__global__ void __launch_bounds__(1024) k_post_ln(const PostLnArgs a) {
    pdl_enter();
    __shared__ float red[32];
    const uint32_t t = blockIdx.x;
    const size_t row = (size_t)t * a.E;
    float *x = a.x + row;
    auto sum_at = [&](uint32_t i, float (&u)[VW]) {
        float xv[VW];
        lds_vec<VW>(x + i, xv);
        if (a.eo) {
#pragma unroll
            for (int e = 0; e < VW; e++) u[e] = 0.0f;
            for (uint32_t j = 0; j < a.top; j++) {
                const float wt = a.wt[(size_t)t * a.top + j];
                float v[VW];
                lds_vec<VW>(a.eo + (size_t)a.slot[(size_t)t * a.top + j] * a.E + i, v);
#pragma unroll
                for (int e = 0; e < VW; e++) u[e] = fmaf(wt, v[e], u[e]);
            }
        } else lds_vec<VW>(a.d + row + i, u);
#pragma unroll
        for (int e = 0; e < VW; e++) u[e] = fmaf(a.alpha, xv[e], u[e]);
    };
    auto store = [&](uint32_t i, const float (&u)[VW], float rinv) {
        float w[VW];
        lds_vec<VW>(a.w + i, w);
#pragma unroll
        for (int e = 0; e < VW; e++) w[e] *= u[e] * rinv;
        stg_vec<VW>(x + i, w);
        if (a.keep) stg_vec<VW>(a.keep + row + i, w);
    };
    float u[NV > 0 ? NV : 1][VW], s = 0.0f;
    if constexpr (NV > 0) {
#pragma unroll
        for (int k = 0; k < NV; k++) {
            const uint32_t i = (threadIdx.x + k * blockDim.x) * VW;
            if (i < a.E) {
                sum_at(i, u[k]);
#pragma unroll
                for (int e = 0; e < VW; e++) s = fmaf(u[k][e], u[k][e], s);
            }
        }
    } else {
        for (uint32_t i = threadIdx.x * VW; i < a.E; i += blockDim.x * VW) {      // a thread reads back only what it wrote
            sum_at(i, u[0]);
            stg_vec<VW>(x + i, u[0]);
#pragma unroll
            for (int e = 0; e < VW; e++) s = fmaf(u[0][e], u[0][e], s);
        }
    }
    s = block_sum(s, red);
    const float rinv = 1.0f / sqrtf(s / (float)a.E + a.eps);
    if constexpr (NV > 0) {
#pragma unroll
        for (int k = 0; k < NV; k++) { const uint32_t i = (threadIdx.x + k * blockDim.x) * VW; if (i < a.E) store(i, u[k], rinv); }
    } else
        for (uint32_t i = threadIdx.x * VW; i < a.E; i += blockDim.x * VW) { lds_vec<VW>(x + i, u[0]); store(i, u[0], rinv); }
}

// ------------------------------------------------------------------------------------------------
// Matrix memory.  Rows of the joint product hold q [H][D] at q0, k [H][D] at k0, v [H][VD] at v0, the output gate [H][VD] at g0 and the two
// raw gates [H] at i0, f0 (biases included).  State per head, fp32: S [VD][D] (a value column is contiguous), n [D], m.
//
// The logs of the gates are added up in double precision: a token's weight depends on the DIFFERENCE of two long sums.  m is rounded to
// fp32 wherever it is kept, and every factor is taken relative to the rounded number, so nothing drifts.
// ------------------------------------------------------------------------------------------------
constexpr uint32_t kMemChunk = 64, kMemDim = 512;
__device__ __forceinline__ float capped_log_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoidf_(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

// grid = H, 1024 threads; a warp takes a chunk, a lane two neighbouring tokens.  With F the sum of f from the chunk's first token on:
// fa[h][t] = F_t, fb[h][t] = i_t - F_t, mt[h][t] = m_t; per chunk fc[h][c] = F at its end, me[h][c] = m before it (me[h][chunks]: at the end)
struct MemGatesArgs { const float *p; uint32_t ld, i0, f0; float cap; float *m; double *fa, *fb, *fc; float *mt, *me; uint32_t T, H, chunks; };
__global__ void __launch_bounds__(1024) k_memory_gates(const MemGatesArgs a) {
    pdl_enter();
    __shared__ double f_s[32], x_s[32];
    __shared__ float in_s[32], m_s;
    const uint32_t h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
    const double ninf = -(double)INFINITY;
    if (threadIdx.x == 0) m_s = a.m[h];
    for (uint32_t base = 0; base < a.chunks; base += 32u) {
        const uint32_t c = base + warp, t0 = c * kMemChunk + 2u * lane;
        double F[2], B[2], R[2];
        float li[2], lf[2];
#pragma unroll
        for (uint32_t j = 0; j < 2; j++) {
            const bool ok = t0 + j < a.T;
            const float *row = a.p + (size_t)(t0 + j) * a.ld + h;
            li[j] = ok ? capped_log_gate(row[a.i0], a.cap) : -INFINITY;
            lf[j] = ok ? log_sigmoidf_(capped_log_gate(row[a.f0], a.cap)) : 0.0f;
        }
        double run = (double)lf[0] + (double)lf[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const double v = __shfl_up_sync(0xffffffffu, run, o); if (lane >= (uint32_t)o) run += v; }
        F[1] = run; F[0] = run - (double)lf[1];
        B[0] = (double)li[0] - F[0]; B[1] = (double)li[1] - F[1];
        double top = fmax(B[0], B[1]);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const double v = __shfl_up_sync(0xffffffffu, top, o); if (lane >= (uint32_t)o) top = fmax(top, v); }
        double before = __shfl_up_sync(0xffffffffu, top, 1);
        if (lane == 0) before = ninf;
        R[0] = fmax(before, B[0]); R[1] = top;
        if (lane == 31) { f_s[warp] = run; x_s[warp] = top; }
        __syncthreads();
        if (threadIdx.x == 0) {
            float m = m_s;
            for (uint32_t w = 0; w < 32u && base + w < a.chunks; w++) { in_s[w] = m; m = (float)(f_s[w] + fmax((double)m, x_s[w])); }
            m_s = m;
        }
        __syncthreads();
        if (c < a.chunks) {
            const double m_in = (double)in_s[warp];
            if (lane == 0) { a.fc[(size_t)h * a.chunks + c] = f_s[warp]; a.me[(size_t)h * (a.chunks + 1u) + c] = in_s[warp]; }
#pragma unroll
            for (uint32_t j = 0; j < 2; j++)
                if (t0 + j < a.T) {
                    const size_t at = (size_t)h * a.T + t0 + j;
                    a.fa[at] = F[j]; a.fb[at] = B[j]; a.mt[at] = (float)(F[j] + fmax(m_in, R[j]));
                }
        }
        __syncthreads();
    }
    if (threadIdx.x == 0) { a.me[(size_t)h * (a.chunks + 1u) + a.chunks] = m_s; a.m[h] = m_s; }
}

// elements at .. at + 3 of a row of n (zeros past its end, and where !ok); vec: 16-byte loads are aligned
__device__ __forceinline__ float4 row4(const float *src, uint32_t at, uint32_t n, bool vec, bool ok) {
    float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (!ok) return v;
    if (vec) { if (at < n) v = *reinterpret_cast<const float4 *>(src + at); return v; }
    if (at < n) v.x = src[at];
    if (at + 1u < n) v.y = src[at + 1u];
    if (at + 2u < n) v.z = src[at + 2u];
    if (at + 3u < n) v.w = src[at + 3u];
    return v;
}
// What every chunk writes, relative to the running maximum at its end:  U_c = sum_s e^(F_C - F_s + i_s - m') k_s v_s^T,  and likewise for n.
// A block makes 64 value columns x 64 key coordinates of one chunk and head, 4 x 4 per thread; the blocks of the first value tile make n
// too.  grid = (value tiles, key tiles, chunks x H), 256 threads.
struct MemWriteArgs { const float *p; uint32_t ld, k0, v0; const double *fb, *fc; const float *me; float *U, *Un; uint32_t T, H, D, VD, chunks; };
__global__ void __launch_bounds__(256, 4) k_memory_writes(const MemWriteArgs a) {
    pdl_enter();
    __shared__ __align__(16) float k_s[kMemChunk][64], v_s[kMemChunk][64];
    __shared__ float w_s[kMemChunk];
    const uint32_t tid = threadIdx.x, tx = tid & 15u, ty = tid >> 4, c = blockIdx.z / a.H, h = blockIdx.z % a.H, col0 = blockIdx.x * 64u, d0 = blockIdx.y * 64u, D = a.D, VD = a.VD;
    const bool vec = ((a.ld | a.k0 | a.v0 | D | VD) & 3u) == 0;
    const double end = a.fc[(size_t)h * a.chunks + c] - (double)a.me[(size_t)h * (a.chunks + 1u) + c + 1u];
#pragma unroll
    for (uint32_t j = 0; j < 4; j++) {
        const uint32_t s = ty + 16u * j, t = c * kMemChunk + s;
        const float *row = a.p + (size_t)t * a.ld;
        const float w = t < a.T ? expf((float)(a.fb[(size_t)h * a.T + t] + end)) : 0.0f;
        const float4 k = row4(row + a.k0 + h * D, d0 + tx * 4u, D, vec, t < a.T), v = row4(row + a.v0 + h * VD, col0 + tx * 4u, VD, vec, t < a.T);
        *reinterpret_cast<float4 *>(&k_s[s][tx * 4u]) = k;
        *reinterpret_cast<float4 *>(&v_s[s][tx * 4u]) = make_float4(v.x * w, v.y * w, v.z * w, v.w * w);
        if (tx == 0) w_s[s] = w;
    }
    __syncthreads();
    float u[4][4] = {}, un = 0.0f;             // u[column][coordinate]
#pragma unroll 8
    for (uint32_t s = 0; s < kMemChunk; s++) {
        const float4 k = *reinterpret_cast<const float4 *>(&k_s[s][tx * 4u]), v = *reinterpret_cast<const float4 *>(&v_s[s][ty * 4u]);
        const float kk[4] = {k.x, k.y, k.z, k.w}, vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (uint32_t i = 0; i < 4; i++)
#pragma unroll
            for (uint32_t j = 0; j < 4; j++) u[i][j] = fmaf(vv[i], kk[j], u[i][j]);
    }
    float *dst = a.U + ((size_t)c * a.H + h) * VD * D;
#pragma unroll
    for (uint32_t i = 0; i < 4; i++) {
        const uint32_t col = col0 + ty * 4u + i, d = d0 + tx * 4u;
        if (col >= VD) continue;
        float *q = dst + (size_t)col * D + d;
        if (vec) { if (d < D) *reinterpret_cast<float4 *>(q) = make_float4(u[i][0], u[i][1], u[i][2], u[i][3]); }
        else {
#pragma unroll
            for (uint32_t e = 0; e < 4; e++) if (d + e < D) q[e] = u[i][e];
        }
    }
    if (blockIdx.x == 0 && tid < 64u && d0 + tid < D) {
#pragma unroll 8
        for (uint32_t s = 0; s < kMemChunk; s++) un = fmaf(w_s[s], k_s[s][tid], un);
        a.Un[((size_t)c * a.H + h) * D + d0 + tid] = un;
    }
}

// In place: U_c becomes the state before chunk c (S, n: the state before the portion, afterwards the one behind it).  A thread walks one
// coordinate of the state (or of n) through the chunks, eight loads in flight.  grid = (blocks over VD D + D, H), 256 threads.
struct MemChainArgs { const double *fc; const float *me; float *S, *n, *U, *Un; uint32_t H, D, VD, chunks; };
__global__ void __launch_bounds__(256) k_memory_chain(const MemChainArgs a) {
    pdl_enter();
    __shared__ float keep_s[256];
    const uint32_t h = blockIdx.y, tid = threadIdx.x, i = blockIdx.x * 256u + tid, nS = a.VD * a.D, total = nS + a.D;
    const bool live = i < total, isS = i < nS;
    float *st = isS ? a.S + (size_t)h * nS + i : a.n + (size_t)h * a.D + (i - nS), *u = isS ? a.U + (size_t)h * nS + i : a.Un + (size_t)h * a.D + (i - nS);
    const size_t step = (size_t)a.H * (isS ? nS : a.D);
    float s = live ? *st : 0.0f;
    for (uint32_t base = 0; base < a.chunks; base += 256u) {
        const uint32_t n = min(256u, a.chunks - base);
        __syncthreads();
        if (tid < n) { const float *me = a.me + (size_t)h * (a.chunks + 1u) + base + tid; keep_s[tid] = (float)exp(a.fc[(size_t)h * a.chunks + base + tid] + (double)me[0] - (double)me[1]); }
        __syncthreads();
        if (!live) continue;
        for (uint32_t c0 = 0; c0 < n; c0 += 8u) {
            float v[8];
#pragma unroll
            for (uint32_t k = 0; k < 8; k++) v[k] = c0 + k < n ? u[(base + c0 + k) * step] : 0.0f;
#pragma unroll
            for (uint32_t k = 0; k < 8; k++)
                if (c0 + k < n) { u[(base + c0 + k) * step] = s; s = fmaf(keep_s[c0 + k], s, v[k]); }
        }
    }
    if (live) *st = s;
}

// All outputs of chunk c = blockIdx.y of head h = blockIdx.z for 64 VJ value columns.  A thread owns 4 tokens x 4 VJ columns.  The key
// coordinates pass in slices of 32: scores q k^T (4 x 4 per thread) and q S of the same slice side by side.  Then the scores get their
// weights e^(F_t - F_s + i_s - m_t) (zero where s > t), and the second product adds the chunk's own values.  256 threads.
struct MemOutArgs { const float *p; uint32_t ld, q0, k0, v0; float qscale; const double *fa, *fb; const float *mt, *me, *Sin, *nin; float *out; uint32_t T, H, D, VD, chunks; };
constexpr uint32_t kMemSlice = 32, kMemLd = kMemSlice + 4, kMemLdp = kMemChunk + 4;
inline size_t memory_out_smem(int vj) {
    const size_t a = (size_t)(2u * kMemChunk + (uint32_t)vj * 64u) * kMemLd + kMemSlice, b = (size_t)kMemChunk * kMemLdp + (size_t)kMemChunk * vj * 64u;
    return (a > b ? a : b) * 4;
}
template <int VJ>
__global__ void __launch_bounds__(256, 2) k_memory_out(const MemOutArgs a) {
    pdl_enter();
    extern __shared__ __align__(16) float sm[];
    constexpr uint32_t VT = VJ * 64u;
    float *q_s = sm, *k_s = q_s + kMemChunk * kMemLd, *S_s = k_s + kMemChunk * kMemLd, *n_s = S_s + VT * kMemLd;      // column j 64 + x 4 + c of S sits in row j 64 + c 16 + x
    float *p_s = sm, *v_s = p_s + kMemChunk * kMemLdp;
    const uint32_t tid = threadIdx.x, tx = tid & 15u, ty = tid >> 4, h = blockIdx.z, c = blockIdx.y, col0 = blockIdx.x * VT, D = a.D, VD = a.VD, t0 = c * kMemChunk;
    const bool vec = ((a.ld | a.q0 | a.k0 | a.v0 | D | VD) & 3u) == 0;
    const float *Sin = a.Sin + ((size_t)c * a.H + h) * VD * D, *nin = a.nin + ((size_t)c * a.H + h) * D;
    float s[4][4] = {}, o[4][VJ * 4] = {}, nq[4] = {};
    float4 qr[2], kr[2], Sr[VJ * 2]; float nr = 0.0f;
    auto fetch = [&](uint32_t d0) {
        const uint32_t e = d0 + (tid & 7u) * 4u;
#pragma unroll
        for (uint32_t j = 0; j < 2; j++) {
            const uint32_t t = t0 + (tid >> 3) + 32u * j;
            const float *row = a.p + (size_t)t * a.ld + h * D;
            qr[j] = row4(row + a.q0, e, D, vec, t < a.T); kr[j] = row4(row + a.k0, e, D, vec, t < a.T);
        }
#pragma unroll
        for (uint32_t j = 0; j < VJ * 2u; j++) { const uint32_t col = col0 + (tid >> 3) + 32u * j; Sr[j] = row4(Sin + (size_t)col * D, e, D, vec, col < VD); }
        if (tid < kMemSlice) nr = d0 + tid < D ? nin[d0 + tid] : 0.0f;
    };
    fetch(0);
    for (uint32_t d0 = 0; d0 < D; d0 += kMemSlice) {
        __syncthreads();
#pragma unroll
        for (uint32_t j = 0; j < 2; j++) {
            const uint32_t at = ((tid >> 3) + 32u * j) * kMemLd + (tid & 7u) * 4u;
            *reinterpret_cast<float4 *>(q_s + at) = make_float4(qr[j].x * a.qscale, qr[j].y * a.qscale, qr[j].z * a.qscale, qr[j].w * a.qscale);
            *reinterpret_cast<float4 *>(k_s + at) = kr[j];
        }
#pragma unroll
        for (uint32_t j = 0; j < VJ * 2u; j++) {
            const uint32_t col = (tid >> 3) + 32u * j, row = (col & ~63u) + (col & 3u) * 16u + ((col & 63u) >> 2);
            *reinterpret_cast<float4 *>(S_s + row * kMemLd + (tid & 7u) * 4u) = Sr[j];
        }
        if (tid < kMemSlice) n_s[tid] = nr;
        __syncthreads();
        if (d0 + kMemSlice < D) fetch(d0 + kMemSlice);
#pragma unroll 2
        for (uint32_t e = 0; e < kMemSlice; e += 4u) {
            float4 qv[4], w[4];
#pragma unroll
            for (uint32_t i = 0; i < 4; i++) { qv[i] = *reinterpret_cast<const float4 *>(q_s + (ty * 4u + i) * kMemLd + e); w[i] = *reinterpret_cast<const float4 *>(k_s + (tx + 16u * i) * kMemLd + e); }
#pragma unroll
            for (uint32_t i = 0; i < 4; i++)
#pragma unroll
                for (uint32_t j = 0; j < 4; j++) s[i][j] = fmaf(qv[i].w, w[j].w, fmaf(qv[i].z, w[j].z, fmaf(qv[i].y, w[j].y, fmaf(qv[i].x, w[j].x, s[i][j]))));
#pragma unroll
            for (uint32_t v = 0; v < VJ; v++) {
#pragma unroll
                for (uint32_t j = 0; j < 4; j++) w[j] = *reinterpret_cast<const float4 *>(S_s + (v * 64u + j * 16u + tx) * kMemLd + e);
#pragma unroll
                for (uint32_t i = 0; i < 4; i++)
#pragma unroll
                    for (uint32_t j = 0; j < 4; j++) { float &x = o[i][v * 4u + j]; x = fmaf(qv[i].w, w[j].w, fmaf(qv[i].z, w[j].z, fmaf(qv[i].y, w[j].y, fmaf(qv[i].x, w[j].x, x)))); }
            }
        }
        if (tx < kMemSlice / 4u) {             // n . q: eight of a row's threads take four coordinates each
            const float4 nn = *reinterpret_cast<const float4 *>(n_s + tx * 4u);
#pragma unroll
            for (uint32_t i = 0; i < 4; i++) { const float4 qv = *reinterpret_cast<const float4 *>(q_s + (ty * 4u + i) * kMemLd + tx * 4u); nq[i] = fmaf(qv.w, nn.w, fmaf(qv.z, nn.z, fmaf(qv.y, nn.y, fmaf(qv.x, nn.x, nq[i])))); }
        }
    }
    __syncthreads();                           // the slices have been read: the weights and the values take their place
    for (uint32_t i = tid; i < kMemChunk * (VT / 4u); i += 256u) {
        const uint32_t k = i / (VT / 4u), e = (i % (VT / 4u)) * 4u;
        *reinterpret_cast<float4 *>(v_s + k * VT + e) = row4(a.p + (size_t)(t0 + k) * a.ld + a.v0 + h * VD, col0 + e, VD, vec, t0 + k < a.T);
    }
    const double *fa = a.fa + (size_t)h * a.T, *fb = a.fb + (size_t)h * a.T;
    const float *mt = a.mt + (size_t)h * a.T;
    const double m_in = (double)a.me[(size_t)h * (a.chunks + 1u) + c];
    double b[4];
#pragma unroll
    for (uint32_t j = 0; j < 4; j++) { const uint32_t t = t0 + tx + 16u * j; b[j] = t < a.T ? fb[t] : 0.0; }
    float inv[4];
#pragma unroll
    for (uint32_t i = 0; i < 4; i++) {
        const uint32_t r = ty * 4u + i, t = min(t0 + r, a.T - 1u);
        const float m = mt[t];
        const double f = fa[t] - (double)m;
        const float before = expf((float)(f + m_in));
        float sum = nq[i] * before;            // threads without coordinates of n hold zero
#pragma unroll
        for (uint32_t j = 0; j < 4; j++) {
            const float v = tx + 16u * j <= r ? s[i][j] * expf((float)(f + b[j])) : 0.0f;
            p_s[r * kMemLdp + tx + 16u * j] = v;
            sum += v;
        }
#pragma unroll
        for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
        inv[i] = 1.0f / (fmaxf(fabsf(sum), expf(-m)) + 1e-6f);
#pragma unroll
        for (uint32_t x = 0; x < VJ * 4u; x++) o[i][x] *= before;
    }
    __syncthreads();
    const uint32_t last = ((ty | 1u) + 1u) * 4u;      // a warp's rows see no later token: the weights are zero there
#pragma unroll 1
    for (uint32_t k = 0; k < last; k += 4u) {
        float4 pv[4];
#pragma unroll
        for (uint32_t i = 0; i < 4; i++) pv[i] = *reinterpret_cast<const float4 *>(p_s + (ty * 4u + i) * kMemLdp + k);
#pragma unroll
        for (uint32_t kk = 0; kk < 4; kk++)
#pragma unroll
            for (uint32_t v = 0; v < VJ; v++) {
                const float4 vv = *reinterpret_cast<const float4 *>(v_s + (k + kk) * VT + v * 64u + tx * 4u);
#pragma unroll
                for (uint32_t i = 0; i < 4; i++) {
                    const float w = kk == 0 ? pv[i].x : kk == 1 ? pv[i].y : kk == 2 ? pv[i].z : pv[i].w;
                    o[i][v * 4] = fmaf(w, vv.x, o[i][v * 4]); o[i][v * 4 + 1] = fmaf(w, vv.y, o[i][v * 4 + 1]);
                    o[i][v * 4 + 2] = fmaf(w, vv.z, o[i][v * 4 + 2]); o[i][v * 4 + 3] = fmaf(w, vv.w, o[i][v * 4 + 3]);
                }
            }
    }
#pragma unroll
    for (uint32_t i = 0; i < 4; i++) {
        const uint32_t t = t0 + ty * 4u + i;
        if (t >= a.T) continue;
        float *dst = a.out + ((size_t)t * a.H + h) * VD + col0;
#pragma unroll
        for (uint32_t v = 0; v < VJ; v++) {
            const uint32_t n = v * 64u + tx * 4u;
            if (vec) { if (col0 + n < VD) *reinterpret_cast<float4 *>(dst + n) = make_float4(o[i][v * 4] * inv[i], o[i][v * 4 + 1] * inv[i], o[i][v * 4 + 2] * inv[i], o[i][v * 4 + 3] * inv[i]); }
            else {
#pragma unroll
                for (uint32_t e = 0; e < 4; e++) if (col0 + n + e < VD) dst[n + e] = o[i][v * 4 + e] * inv[i];
            }
        }
    }
}

// Short portions (T <= kGemvMaxM): a cluster of blocks per head, each with a share of its value columns (8 lanes per column, the column's
// state in registers), from the joint product's rows to  o / rms(o) gain sigmoid(g).  Every block walks n and the gates itself (one warp);
// the first block of the cluster writes n and m back once all blocks have read them.  The blocks exchange their columns' sums of squares.
constexpr uint32_t kMemBlocks = 8, kMemThreads = 512;
__host__ __device__ inline uint32_t memory_step_blocks(uint32_t VD) { return VD >= 128u ? 8u : VD >= 64u ? 4u : VD >= 32u ? 2u : 1u; }
__host__ __device__ inline uint32_t memory_step_cols(uint32_t VD) { const uint32_t n = memory_step_blocks(VD); return ((VD + n - 1u) / n + 3u) & ~3u; }
struct MemStepArgs { const float *p; uint32_t ld, q0, k0, v0, g0, i0, f0; float cap, qscale, eps; const float *gain; float *S, *n, *m, *out; uint32_t T, H, D, VD; };
inline size_t memory_step_smem(int dch, uint32_t VD) { return ((size_t)2 * kGemvMaxM * (uint32_t)dch * 32u + (size_t)2 * kGemvMaxM * memory_step_cols(VD)) * 4; }      // dch: the instance's, DCH
template <int DCH>
__global__ void __launch_bounds__(kMemThreads) k_memory_step(const MemStepArgs a) {
    pdl_launch_next();
    cluster_arrive();                          // waited for before the first access to another block's shared memory
    pdl_wait();
    constexpr uint32_t DP = DCH * 32u;
    extern __shared__ __align__(16) float sm[];
    __shared__ float keep_s[kGemvMaxM], write_s[kGemvMaxM], inv_s[kGemvMaxM], ss_s[kGemvMaxM][kMemBlocks];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, sub = lane & 7u, nw = blockDim.x >> 5, h = blockIdx.y, D = a.D, VD = a.VD, T = a.T;
    const uint32_t CB = memory_step_cols(VD), col_lo = min(VD, blockIdx.x * CB), nc = min(VD, col_lo + CB) - col_lo, groups = blockDim.x >> 3;      // this block's value columns
    float *q_s = sm, *k_s = q_s + kGemvMaxM * DP, *o_s = k_s + kGemvMaxM * DP, *gate_s = o_s + kGemvMaxM * CB;
    const bool dvec = (D & 3u) == 0;
    float S[DCH][4], v_r[kGemvMaxM];
    auto load_column = [&](uint32_t j) {       // a column's state and its values of every token; j: column of this block
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
        for (uint32_t t = 0; t < kGemvMaxM; t++) v_r[t] = (t < T && j < nc) ? a.p[(size_t)t * a.ld + a.v0 + h * VD + col_lo + j] : 0.0f;
    };
    load_column(tid >> 3);                     // in flight while the vectors and gates are made
    for (uint32_t i = tid; i < T * nc; i += blockDim.x) { const uint32_t t = i / nc, j = i % nc; gate_s[t * CB + j] = sigmoidf_(a.p[(size_t)t * a.ld + a.g0 + h * VD + col_lo + j]) * a.gain[h * VD + col_lo + j]; }
    for (uint32_t i = tid; i < T * DP; i += blockDim.x) {
        const uint32_t t = i / DP, d = i % DP;
        const float *row = a.p + (size_t)t * a.ld + h * D + d;
        q_s[i] = d < D ? row[a.q0] * a.qscale : 0.0f; k_s[i] = d < D ? row[a.k0] : 0.0f;
    }
    float nr[DCH]; double m = 0.0;
    if (warp == nw - 1u) {
#pragma unroll
        for (int c = 0; c < DCH; c++) { const uint32_t d = lane + 32u * c; nr[c] = d < D ? a.n[(size_t)h * D + d] : 0.0f; }
        m = (double)a.m[h];
        for (uint32_t t = 0; t < T; t++) {
            const float *row = a.p + (size_t)t * a.ld + h;
            const double li = (double)capped_log_gate(row[a.i0], a.cap), stay = (double)log_sigmoidf_(capped_log_gate(row[a.f0], a.cap)) + m;
            const float mf = (float)fmax(stay, li), keep = (float)exp(stay - (double)mf), write = (float)exp(li - (double)mf);      // double, rounded once: a state takes thousands of these factors
            m = (double)mf;
            float nq = 0.0f;
            const float *q = a.p + (size_t)t * a.ld + a.q0 + h * D, *k = a.p + (size_t)t * a.ld + a.k0 + h * D;
#pragma unroll
            for (int c = 0; c < DCH; c++) { const uint32_t d = lane + 32u * c; if (d < D) { nr[c] = fmaf(write, k[d], keep * nr[c]); nq = fmaf(nr[c], q[d] * a.qscale, nq); } }
            nq = warp_sum(nq);
            if (lane == 0) { keep_s[t] = keep; write_s[t] = write; inv_s[t] = 1.0f / (fmaxf(fabsf(nq), expf(-mf)) + 1e-6f); }
        }
    }
    __syncthreads();
    for (uint32_t c0 = 0; c0 < nc; c0 += groups) {
        const uint32_t j = c0 + (tid >> 3);
        if (c0) load_column(j);
#pragma unroll
        for (uint32_t t = 0; t < kGemvMaxM; t++) {
            if (t >= T) break;
            const float keep = keep_s[t], wv = write_s[t] * v_r[t];
            float pq = 0.0f;
#pragma unroll
            for (int c = 0; c < DCH; c++) {
                const uint32_t d = t * DP + (sub + 8u * c) * 4u;
                const float4 kv = *reinterpret_cast<const float4 *>(k_s + d), qv = *reinterpret_cast<const float4 *>(q_s + d);
                S[c][0] = fmaf(kv.x, wv, keep * S[c][0]); S[c][1] = fmaf(kv.y, wv, keep * S[c][1]); S[c][2] = fmaf(kv.z, wv, keep * S[c][2]); S[c][3] = fmaf(kv.w, wv, keep * S[c][3]);
                pq = fmaf(S[c][3], qv.w, fmaf(S[c][2], qv.z, fmaf(S[c][1], qv.y, fmaf(S[c][0], qv.x, pq))));
            }
#pragma unroll
            for (int off = 4; off > 0; off >>= 1) pq += __shfl_xor_sync(0xffffffffu, pq, off);
            if (sub == 0 && j < nc) o_s[t * CB + j] = pq * inv_s[t];
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
    cluster_wait();                            // every block of the cluster runs
    for (uint32_t t = warp; t < T; t += nw) {  // this block's share of the head's sum of squares, to every block of the head
        float s = 0.0f;
        for (uint32_t j = lane; j < nc; j += 32u) s = fmaf(o_s[t * CB + j], o_s[t * CB + j], s);
        s = warp_sum(s);
        if (lane < gridDim.x) st_cluster(&ss_s[t][blockIdx.x], lane, s);
    }
    __syncwarp();
    cluster_arrive();
    cluster_wait();                            // every block of the head has read n and m
    if (blockIdx.x == 0 && warp == nw - 1u) {
#pragma unroll
        for (int c = 0; c < DCH; c++) { const uint32_t d = lane + 32u * c; if (d < D) a.n[(size_t)h * D + d] = nr[c]; }
        if (lane == 0) a.m[h] = (float)m;
    }
    for (uint32_t i = tid; i < T * nc; i += blockDim.x) {
        const uint32_t t = i / nc, j = i % nc;
        float s = 0.0f;
        for (uint32_t r = 0; r < gridDim.x; r++) s += ss_s[t][r];
        a.out[((size_t)t * a.H + h) * VD + col_lo + j] = o_s[t * CB + j] / sqrtf(s / (float)VD + a.eps) * gate_s[t * CB + j];
    }
}

}  // namespace lm
}  // namespace nb
