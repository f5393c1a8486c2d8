// Kernels of the MoE + MLA decoder (a mixture-of-experts FFN behind multi-head latent attention),
// one token per step.  The reference has neither (no router, expert or latent-cache code anywhere
// in it): the model is defined by this repository (include/cuda_decode.h, cd_moe_config) and what
// it shares with the dense model - RMSNorm (lib.rs:1354-1378), interleaved-pair RoPE
// (lib.rs:1392-1408), SwiGLU (lib.rs:1504-1513), the scaled residuals (lib.rs:1491-1502) - is
// computed exactly as there.
//
// Per layer (H heads, C latent width, R RoPE width, N / V per-head no-position / value widths):
//   gemv_tma_kernel      RMSNorm + [q | latent | rope key] = W_qa xn            (the dense GEMV, plain store)
//   mla_post_kernel      RoPE on the q heads' RoPE parts and on the key; RMSNorm of the latent; the
//                        cache row [latent | rope key] into its page; per head the absorbed query
//                        q'_h = W_uk_h^T q_nope_h, so that a score is one 576-wide dot with a cache row
//   mla_attn_kernel      split over cached positions: every CTA reads its positions once for all heads
//                        (the cache is shared by the heads), running softmax, partial latent sums
//   mla_out_kernel       merges the slices (fixed order) and applies W_uv_h: the head's output
//   gemv_tma_kernel      Wo + scaled residual
//   moe_router_kernel    RMSNorm, router logits, softmax over all experts, top-k (ties: lower index)
//   moe_w13_kernel       gate = silu(xn W1) * (xn W3) * p for the chosen experts and the shared ones
//   moe_w2_kernel        x = x2 + alpha * sum over experts of W2 gate; expert parallel: the rank's partial
//                        sum is pushed to every rank's inbox instead (the dense model's all-reduce)
// All of them are HBM-bound streams of weight rows (or cache rows) with fp32 accumulation.
#pragma once
#include "common.cuh"

namespace cd {

constexpr int MLA_MAX_HEADS = 16;   // heads whose state one attention CTA keeps: more heads go to further CTAs
constexpr int MLA_MAX_COLS = 512;   // latent columns it accumulates: wider latents likewise
constexpr int MLA_TILE = 16;        // cached positions per attention tile

// dot of one weight row (K elements, storage WT) with x (fp32, shared memory): the lanes of a warp take
// 16-byte chunks round robin; result valid in every lane
template <typename WT> __device__ inline float warp_row_dot(const WT* __restrict__ row, const float* xs, int K, int lane) {
    constexpr int EPC = Elem<WT>::EPC;
    float a = 0.0f;
#pragma unroll 4
    for (int c = lane; c < K / EPC; c += 32) {
        const uint4 w = ldg_stream(reinterpret_cast<const char*>(row) + (size_t)c * 16);
        float f[EPC];
        Elem<WT>::unpack(w, f);
#pragma unroll
        for (int e = 0; e < EPC; e += 4) {  // x in 16-byte pieces: one shared-memory transaction per four elements
            const float4 x4 = *reinterpret_cast<const float4*>(xs + c * EPC + e);
            a = fmaf(f[e], x4.x, a); a = fmaf(f[e + 1], x4.y, a); a = fmaf(f[e + 2], x4.z, a); a = fmaf(f[e + 3], x4.w, a);
        }
    }
    return warp_sum(a);
}

// The same for NR rows `stride` elements apart: the loads of all rows are in flight together (a single row per
// warp is bound by one memory latency per row)
template <typename WT, int NR>
__device__ inline void warp_rows_dot(const WT* __restrict__ rows, size_t stride, const float* xs, int K, int lane, float (&out)[NR]) {
    constexpr int EPC = Elem<WT>::EPC;
    float a[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) a[r] = 0.0f;
#pragma unroll 2
    for (int c = lane; c < K / EPC; c += 32) {
        uint4 w[NR];
#pragma unroll
        for (int r = 0; r < NR; ++r) w[r] = ldg_stream(reinterpret_cast<const char*>(rows + (size_t)r * stride) + (size_t)c * 16);
        float x[EPC];
#pragma unroll
        for (int e = 0; e < EPC; e += 4) {
            const float4 x4 = *reinterpret_cast<const float4*>(xs + c * EPC + e);
            x[e] = x4.x; x[e + 1] = x4.y; x[e + 2] = x4.z; x[e + 3] = x4.w;
        }
#pragma unroll
        for (int r = 0; r < NR; ++r) {
            float f[EPC];
            Elem<WT>::unpack(w[r], f);
#pragma unroll
            for (int e = 0; e < EPC; ++e) a[r] = fmaf(f[e], x[e], a[r]);
        }
    }
#pragma unroll
    for (int r = 0; r < NR; ++r) out[r] = warp_sum(a[r]);
}

// Widths as stored: the cache row is [latent | rope], a row of the absorbed-key matrix has nope elements (each a multiple of
// 16 bytes where the kernels ask for it, zeros behind the model's own widths latent_n, rope_n, nope_n, which are those of
// the projection row [heads (nope_n + rope_n) | latent_n | rope_n]).
struct MlaDims {
    int heads, latent, rope, nope, vdim, page_tokens;
    int latent_n, rope_n, nope_n;
    int rot_dims;        // rotated entries of the rope part, the first ones
    int window;          // positions seen, itself included; 0: all
    float eps;           // of the latent's norm
    __host__ __device__ int row() const { return latent + rope; }
    __host__ __device__ int head_blocks() const { return (heads + MLA_MAX_HEADS - 1) / MLA_MAX_HEADS; }
    __host__ __device__ int col_blocks() const { return (latent + MLA_MAX_COLS - 1) / MLA_MAX_COLS; }
    // the attention kernels' split of the visible positions: slice s holds first .. first + per - 1 (up to pos)
    __device__ int first_seen(int pos) const { return window > 0 ? max(0, pos - window + 1) : 0; }
    __device__ int slice(int pos, int nsplit, int tile) const {
        const int per = (pos + 1 - first_seen(pos) + nsplit - 1) / nsplit;
        return (per + tile - 1) / tile * tile;
    }
};

// cos and sin of a position's k-th rotation: from a table [position][dims / 2], or worked out from the angular frequencies
// (angle and its reduction in double, so that far positions keep their fp32 accuracy)
struct Rotation {
    const float2* table;
    const double* freq;
    int dims;
    __device__ float2 at(int pos, int k) const {
        if (table != nullptr) return table[(size_t)pos * (dims / 2) + k];
        const double turns = (double)pos * freq[k] * 0.15915494309189533577;  // 1 / (2 pi)
        const float a = (float)((turns - rint(turns)) * 6.283185307179586477);
        float2 cs;
        sincosf(a, &cs.y, &cs.x);
        return cs;
    }
    // all of a position's rotations into shared memory (whole CTA; the caller's barrier publishes them)
    __device__ void fill(float2* cs, int pos) const {
        for (int k = threadIdx.x; k < dims / 2; k += blockDim.x) cs[k] = at(pos, k);
    }
    // entry d of a vector whose raw entries get(i) returns; cs(k) is the k-th rotation
    template <class Cs, class Get> __device__ float entry(int d, Cs cs_of, Get get) const {
        if (d >= dims) return get(d);
        const float2 cs = cs_of(d >> 1);
        const float u = get(d & ~1), v = get(d | 1);
        return (d & 1) ? v * cs.x + u * cs.y : u * cs.x - v * cs.y;
    }
};

// ---------------------------------------------------------------------- after the q | latent | key GEMV
// CTAs of 128 threads.  The first ceil(heads * C / 128): one thread per row (h, c) of the absorbed-key matrix,
// q'_h[c] = sum_d W_uk[c, h N + d] q_nope_h[d] (a row is N elements: every thread has its whole row in flight); the next
// ceil(heads * R / 256): RoPE on the heads' RoPE parts of q, a pair per thread; the last CTA: the cache row of this
// position [rmsnorm(latent) | rope(key)].  qabs[h] = [q'_h (C) | rope(q_rope_h) (R)].
template <typename WT, typename KT>
__global__ void __launch_bounds__(128)
mla_post_kernel(const float* __restrict__ qa, const WT* __restrict__ wuk_t, const float* __restrict__ gamma_kv, Rotation rot,
                const int* __restrict__ page_table, const DevState* st, KT* __restrict__ lat_pool, float* __restrict__ qabs, KT* __restrict__ qsplit,
                MlaDims d) {
    extern __shared__ float sm[];  // [heads * N] the no-position parts of q (absorb CTAs) or [C] the raw latent (last CTA)
    __shared__ float red[32];
    constexpr int EPC = Elem<WT>::EPC;
    const int tid = threadIdx.x;
    const int H = d.heads, C = d.latent, R = d.rope, N = d.nope, QH = d.nope_n + d.rope_n;
    // qsplit (16-bit cache only): per block of 16 heads [2][16][C + R], the 16-bit head of qabs and the 16-bit remainder, the
    // tensor-core attention's A operand
    auto put = [&](int h, int k, float v) {
        qabs[(size_t)h * (C + R) + k] = v;
        if (qsplit != nullptr) {
            KT* q = qsplit + (size_t)((h >> 4) * 32 + (h & 15)) * (C + R) + k;
            const KT hi = Elem<KT>::from_f32(v);
            *q = hi;
            q[(size_t)16 * (C + R)] = Elem<KT>::from_f32(v - Elem<KT>::to_f32(hi));
        }
    };
    const int n_absorb = (H * C + 127) / 128;
    if ((int)blockIdx.x < n_absorb) {
        const int r = min((int)(blockIdx.x * blockDim.x) + tid, H * C - 1);  // row (h, c)
        const char* row = reinterpret_cast<const char*>(wuk_t + (size_t)r * N);
        constexpr int PRE = 16;  // chunks of the row requested before anything else (a whole 128-wide 16-bit row)
        uint4 w[PRE];
#pragma unroll
        for (int j = 0; j < PRE; ++j) w[j] = j < N / EPC ? ldg_stream(row + (size_t)j * 16) : make_uint4(0, 0, 0, 0);
        pdl_wait();  // the weights above do not depend on the previous kernel, q does
        pdl_launch_dependents();
        // only the heads this CTA's rows belong to
        const int h0 = (int)(blockIdx.x * blockDim.x) / C, h1 = min((int)((blockIdx.x + 1) * blockDim.x - 1) / C, H - 1);
        for (int i = tid; i < (h1 - h0 + 1) * N; i += blockDim.x) sm[i] = i % N < d.nope_n ? __ldcg(qa + (size_t)(h0 + i / N) * QH + (i % N)) : 0.0f;
        __syncthreads();
        if ((int)(blockIdx.x * blockDim.x) + tid >= H * C) return;
        const int h = r / C;
        const float* qn = sm + (h - h0) * N;
        float acc = 0.0f;
#pragma unroll
        for (int j = 0; j < PRE; ++j) {
            if (j < N / EPC) {
                float f[EPC];
                Elem<WT>::unpack(w[j], f);
#pragma unroll
                for (int e = 0; e < EPC; ++e) acc = fmaf(f[e], qn[j * EPC + e], acc);
            }
        }
        for (int c0 = PRE; c0 < N / EPC; c0 += 8) {  // wider rows: eight more chunks in flight at a time
            uint4 v[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = c0 + j < N / EPC ? ldg_stream(row + (size_t)(c0 + j) * 16) : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                if (c0 + j < N / EPC) {
                    float f[EPC];
                    Elem<WT>::unpack(v[j], f);
#pragma unroll
                    for (int e = 0; e < EPC; ++e) acc = fmaf(f[e], qn[(c0 + j) * EPC + e], acc);
                }
            }
        }
        put(h, r % C, acc);
        return;
    }
    pdl_wait();
    pdl_launch_dependents();
    const int pos = __ldcg(&st->pos);
    if (blockIdx.x + 1 < gridDim.x) {  // rotation of q's part of it
        const int i = 2 * (((int)blockIdx.x - n_absorb) * (int)blockDim.x + tid), h = i / R, k = i % R;
        if (i >= H * R) return;
        const float* q = qa + (size_t)h * QH + d.nope_n;
        float u = k < d.rope_n ? __ldcg(q + k) : 0.0f, v = k + 1 < d.rope_n ? __ldcg(q + k + 1) : 0.0f;
        if (k < rot.dims) {
            const float2 cs = rot.at(pos, k >> 1);
            const float t = u * cs.x - v * cs.y;
            v = v * cs.x + u * cs.y;
            u = t;
        }
        put(h, C + k, u);
        put(h, C + k + 1, v);
        return;
    }
    // the cache row: normed latent | rotated key
    const float* craw = qa + (size_t)H * QH;
    float2* cs = reinterpret_cast<float2*>(sm + ((C + 1) & ~1));  // [dims / 2]
    auto cs_of = [&](int k) { return cs[k]; };
    float ss = 0.0f;
#pragma unroll 8
    for (int i = tid; i < d.latent_n; i += blockDim.x) {
        const float v = __ldcg(craw + i);
        sm[i] = v;
        ss += v * v;
    }
    rot.fill(cs, pos);
    const float tot = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(tot * (1.0f / (float)d.latent_n) + d.eps);
    const int page = page_table[pos / d.page_tokens], off = pos % d.page_tokens;
    KT* row = lat_pool + ((size_t)page * d.page_tokens + off) * (C + R);
    for (int i = tid; i < C; i += blockDim.x) row[i] = Elem<KT>::from_f32(i < d.latent_n ? sm[i] * inv * gamma_kv[i] : 0.0f);
    for (int i = tid; i < R; i += blockDim.x)
        row[C + i] = Elem<KT>::from_f32(i < d.rope_n ? rot.entry(i, cs_of, [&](int j) { return __ldcg(craw + d.latent_n + j); }) : 0.0f);
}
__host__ __device__ inline size_t mla_post_smem_floats(const MlaDims& d) { return max((128 / d.latent + 2) * d.nope, d.latent + 2 + d.rope); }
__host__ __device__ inline int mla_post_ctas(const MlaDims& d) { return (d.heads * d.latent + 127) / 128 + (d.heads * d.rope + 255) / 256 + 1; }

// ---------------------------------------------------------------------- latent attention, one slice of cached positions per CTA
// score_h(t) = qabs_h . row(t) * scale over the C + R wide cache row; out_h = sum_t p_h(t) row(t)[0 .. C).
// Shared memory: qs [H][W + 1], rows [MLA_TILE][W + 1] (W = C + R; the pad keeps the columns on
// different banks), sc [H][MLA_TILE], state [3][H].  256 threads; thread t owns latent dimensions
// t and t + 256 of every head.  grid = (slices, blocks of 16 heads, blocks of 512 latent columns).
__host__ __device__ inline size_t mla_attn_smem_floats(const MlaDims& d) {
    const size_t h = min(d.heads, MLA_MAX_HEADS), w = d.row();
    return h * (w + 1) + (size_t)MLA_TILE * (w + 1) + h * MLA_TILE + 3 * h;
}
template <typename KT>
__global__ void __launch_bounds__(256)
mla_attn_kernel(const float* __restrict__ qabs, const KT* __restrict__ lat_pool, const int* __restrict__ page_table, const DevState* st,
                float* __restrict__ part_acc, float* __restrict__ part_ml, MlaDims d, int nsplit, float scale) {
    extern __shared__ float sm[];
    constexpr float NEG = -3.402823466e+38f;
    const int h0 = blockIdx.y * MLA_MAX_HEADS, col0 = blockIdx.z * MLA_MAX_COLS;
    const int tid = threadIdx.x, H = min(d.heads - h0, MLA_MAX_HEADS), C = min(d.latent - col0, MLA_MAX_COLS), W = d.latent + d.rope, LD = W + 1, s = blockIdx.x;
    float* qs = sm;                          // [H][LD]
    float* rows = qs + (size_t)H * LD;       // [MLA_TILE][LD]
    float* sc = rows + (size_t)MLA_TILE * LD;  // [H][MLA_TILE] probabilities of the tile
    float* mrun = sc + H * MLA_TILE;         // [H] running maximum
    float* lrun = mrun + H;                  // [H] running sum
    float* corr = lrun + H;                  // [H] rescale factor of the tile
    pdl_wait();
    pdl_launch_dependents();  // after the wait: at most this kernel and the next one overlap
    const int pos = __ldcg(&st->pos), per = d.slice(pos, nsplit, MLA_TILE);
    const int t0 = d.first_seen(pos) + s * per, t1 = min(pos + 1, t0 + per);
    for (int i = tid; i < H * W; i += 256) qs[(i / W) * LD + (i % W)] = __ldcg(qabs + (size_t)h0 * W + i);
    if (tid < H) { mrun[tid] = NEG; lrun[tid] = 0.0f; }
    float acc[MLA_MAX_HEADS][2];
#pragma unroll
    for (int h = 0; h < MLA_MAX_HEADS; ++h) acc[h][0] = acc[h][1] = 0.0f;
    __syncthreads();
    for (int tb = t0; tb < t1; tb += MLA_TILE) {
        const int nt = min(MLA_TILE, t1 - tb);
        for (int i = tid; i < nt * W; i += 256) {  // the tile's cache rows, widened to fp32
            const int j = i / W, k = i % W, t = tb + j;
            const int page = page_table[t / d.page_tokens], off = t % d.page_tokens;
            rows[j * LD + k] = Elem<KT>::to_f32(__ldcg(lat_pool + ((size_t)page * d.page_tokens + off) * W + k));  // the newest row was written this token
        }
        __syncthreads();
        for (int base = 0; base < H * MLA_TILE; base += 256) {  // one (head, position) score per thread; whole warps take part in the shuffles
            const int item = base + tid;
            const bool live = item < H * MLA_TILE;
            const int h = live ? item / MLA_TILE : 0, j = item % MLA_TILE;
            float v = NEG;
            if (live && j < nt) {
                const float* q = qs + h * LD;
                const float* r = rows + j * LD;
                float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
                int k = 0;
                for (; k + 4 <= W; k += 4) {
                    a0 = fmaf(q[k], r[k], a0); a1 = fmaf(q[k + 1], r[k + 1], a1);
                    a2 = fmaf(q[k + 2], r[k + 2], a2); a3 = fmaf(q[k + 3], r[k + 3], a3);
                }
                for (; k < W; ++k) a0 = fmaf(q[k], r[k], a0);
                v = ((a0 + a1) + (a2 + a3)) * scale;
            }
            // the MLA_TILE lanes of a head sit side by side in one warp: maximum and sum by shuffles
            float mx = v;
#pragma unroll
            for (int o = MLA_TILE / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mold = mrun[h], mnew = fmaxf(mold, mx);
            const float p = (live && j < nt) ? expf(v - mnew) : 0.0f;
            float ps = p;
#pragma unroll
            for (int o = MLA_TILE / 2; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
            if (live) sc[item] = p;
            __syncwarp();
            if (live && j == 0) {
                const float c = expf(mold - mnew);
                corr[h] = c;
                lrun[h] = lrun[h] * c + ps;
                mrun[h] = mnew;
            }
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < MLA_MAX_HEADS; ++h) {
            if (h < H) {
                const float c = corr[h];
                float a0 = acc[h][0] * c, a1 = acc[h][1] * c;
                for (int j = 0; j < nt; ++j) {
                    const float p = sc[h * MLA_TILE + j];
                    if (tid < C) a0 = fmaf(p, rows[j * LD + col0 + tid], a0);
                    if (tid + 256 < C) a1 = fmaf(p, rows[j * LD + col0 + tid + 256], a1);
                }
                acc[h][0] = a0; acc[h][1] = a1;
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int h = 0; h < MLA_MAX_HEADS; ++h) {
        if (h < H) {
            float* pa = part_acc + ((size_t)s * d.heads + h0 + h) * d.latent + col0;
            if (tid < C) pa[tid] = acc[h][0];
            if (tid + 256 < C) pa[tid + 256] = acc[h][1];
        }
    }
    if (tid < H) {
        part_ml[((size_t)s * d.heads + h0 + tid) * 2 + 0] = mrun[tid];
        part_ml[((size_t)s * d.heads + h0 + tid) * 2 + 1] = lrun[tid];
    }
}

// ---------------------------------------------------------------------- merge the slices, apply W_uv: grid = (heads, ceil(V / 32))
template <typename WT>
__global__ void __launch_bounds__(256)
mla_out_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml, const WT* __restrict__ wuv_t, float* __restrict__ attn_out,
               const DevState* st, MlaDims d, int nsplit_max, int tile) {
    extern __shared__ float sm[];  // [C] the head's latent-space output, then [nsplit] slice weights
    constexpr float NEG = -3.402823466e+38f;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;  // eight warps
    const int H = d.heads, C = d.latent, V = d.vdim, h = blockIdx.x;
    float* lat = sm;
    float* wsl = sm + C;
    __shared__ float s_inv;
    pdl_wait();
    pdl_launch_dependents();  // after the wait: at most this kernel and the next one overlap
    // the attention kernel's split of this context: slices of `per` positions, the first `nsplit` of them hold any
    const int pos = __ldcg(&st->pos), per = d.slice(pos, nsplit_max, tile);
    const int nsplit = (pos - d.first_seen(pos)) / per + 1;
    if (warp == 0) {
        float M = NEG;
        for (int s = lane; s < nsplit; s += 32) {
            const float2 ml = __ldcg(reinterpret_cast<const float2*>(part_ml) + (size_t)s * H + h);
            if (ml.y > 0.0f) M = fmaxf(M, ml.x);
        }
        M = warp_max(M);
        for (int s = lane; s < nsplit; s += 32) {
            const float2 ml = __ldcg(reinterpret_cast<const float2*>(part_ml) + (size_t)s * H + h);
            wsl[s] = ml.y > 0.0f ? expf(ml.x - M) : 0.0f;
        }
        // the slices' sums are added in slice order by one lane, so the result does not depend on the lane count
        __syncwarp();
        if (lane == 0) {
            float tot = 0.0f;
            for (int s = 0; s < nsplit; ++s) {
                const float2 ml = __ldcg(reinterpret_cast<const float2*>(part_ml) + (size_t)s * H + h);
                tot += ml.y * wsl[s];
            }
            s_inv = tot > 0.0f ? 1.0f / tot : 0.0f;
        }
    }
    __syncthreads();
    for (int c = 2 * tid; c < C; c += 2 * blockDim.x) {  // C is even
        float a0 = 0.0f, a1 = 0.0f;
#pragma unroll 16
        for (int s = 0; s < nsplit; ++s) {  // slice order
            const float2 v = __ldcg(reinterpret_cast<const float2*>(part_acc + ((size_t)s * H + h) * C + c));
            a0 = fmaf(v.x, wsl[s], a0);
            a1 = fmaf(v.y, wsl[s], a1);
        }
        lat[c] = a0 * s_inv;
        lat[c + 1] = a1 * s_inv;
    }
    __syncthreads();
    // this CTA's 32 output rows of the head: four rows per warp, their loads in flight together
    const int dv0 = blockIdx.y * 32 + warp * 4;
    if (dv0 + 4 <= V) {
        float y[4];
        warp_rows_dot<WT, 4>(wuv_t + ((size_t)h * V + dv0) * C, (size_t)C, lat, C, lane, y);
        if (lane < 4) attn_out[(size_t)h * V + dv0 + lane] = lane == 0 ? y[0] : lane == 1 ? y[1] : lane == 2 ? y[2] : y[3];
    } else {
        for (int dv = dv0; dv < V; ++dv) {
            const float v = warp_row_dot<WT>(wuv_t + ((size_t)h * V + dv) * C, lat, C, lane);
            if (lane == 0) attn_out[(size_t)h * V + dv] = v;
        }
    }
}

// ---------------------------------------------------------------------- latent attention on the tensor cores
// The absorbed form is a GEMM with M = heads: scores S[h, t] = qabs[h, :] . row(t) over the C + R wide
// cache row, output O[h, :] = sum_t p[h, t] row(t)[0 .. C).  mma.sync m16n8k16 with fp32 accumulation;
// the fp32 operands (q, p) are split into a 16-bit head and a 16-bit remainder (two MMAs), so only the
// cache itself carries its storage rounding.  One CTA of four warps per slice of cached positions, 64
// positions at a time: the tile's rows arrive by one bulk copy each (row stride padded by 16 bytes: ldmatrix
// without bank conflicts); warp w scores positions 16 w .. 16 w + 15, then owns latent columns
// CW w .. CW w + CW - 1 of every head (CW = 128; 64 and 32 for narrower latents).  grid = (slices, blocks of 16 heads, blocks
// of 4 CW latent columns).  Geometry: 16-bit cache, C and R multiples of 16.
constexpr int MLA_MMA_TILE = 64, MLA_MMA_THREADS = 128;

template <typename KT> struct Mma16;
template <> struct Mma16<__half> {
    __device__ static inline void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
        asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                     : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
    }
};
template <> struct Mma16<__nv_bfloat16> {
    __device__ static inline void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
        asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                     : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
    }
};
__device__ inline void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ inline void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

__host__ __device__ inline size_t mla_mma_smem_bytes(int W) {
    const size_t ldb = (size_t)W * 2 + 16;
    return (size_t)(MLA_MMA_TILE + 32) * ldb            // rows, q head, q remainder
           + (size_t)16 * (MLA_MMA_TILE + 1) * 4         // scores
           + (size_t)2 * 16 * (MLA_MMA_TILE + 8) * 2     // p head, p remainder
           + 3 * 16 * 4 + 16;                            // running max, sum, rescale; mbarrier
}

template <typename KT, int CW>
__global__ void __launch_bounds__(MLA_MMA_THREADS)
mla_attn_mma_kernel(const KT* __restrict__ qsplit, const KT* __restrict__ lat_pool, const int* __restrict__ page_table, const DevState* st,
                    float* __restrict__ part_acc, float* __restrict__ part_ml, MlaDims d, int nsplit, float scale, int* err) {
    extern __shared__ __align__(128) unsigned char smraw[];
    constexpr float NEG = -3.402823466e+38f;
    constexpr int T = MLA_MMA_TILE, LDS = T + 1, LDP = T + 8;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h0 = blockIdx.y * MLA_MAX_HEADS, H = min(d.heads - h0, MLA_MAX_HEADS), C = d.latent;
    const int W = d.latent + d.rope, s = blockIdx.x, col0 = (blockIdx.z * 4 + warp) * CW;  // this warp's latent columns
    qsplit += (size_t)blockIdx.y * 32 * W;
    const uint32_t LDB = (uint32_t)W * 2u + 16u;
    unsigned char* rows_p = smraw;                                   // [T][LDB]
    unsigned char* qh_p = rows_p + (size_t)T * LDB;                  // [16][LDB]
    unsigned char* ql_p = qh_p + (size_t)16 * LDB;                   // [16][LDB], directly behind qh
    float* sc = reinterpret_cast<float*>(ql_p + (size_t)16 * LDB);   // [16][LDS]
    KT* ph = reinterpret_cast<KT*>(sc + 16 * LDS);                   // [16][LDP]
    KT* pl = ph + 16 * LDP;                                          // [16][LDP]
    float* mrun = reinterpret_cast<float*>(pl + 16 * LDP);           // [16]
    float* lrun = mrun + 16;
    float* corr = lrun + 16;
    uint64_t* bar_p = reinterpret_cast<uint64_t*>(corr + 16);
    const uint32_t rows = smem_addr(rows_p), qh = smem_addr(qh_p), ql = smem_addr(ql_p), bar = smem_addr(bar_p);
    const uint32_t pha = smem_addr(ph), pla = smem_addr(pl);

    pdl_wait();
    pdl_launch_dependents();  // after the wait: at most this kernel and the next one overlap
    const int pos = __ldcg(&st->pos), per = d.slice(pos, nsplit, T);
    const int t0 = d.first_seen(pos) + s * per, t1 = min(pos + 1, t0 + per);
    if (t0 >= t1) return;  // a slice past the context: mla_out_kernel merges the slices that hold positions only
    if (tid == 0) {
        mbar_init(bar, 1);
        mbar_fence_init();
    }
    if (tid < 16) { mrun[tid] = NEG; lrun[tid] = 0.0f; corr[tid] = 0.0f; }
    __syncthreads();
    auto fetch = [&](int tb, bool with_q) {  // warp 0: one bulk copy per cached row of the tile (and per row of q)
        const int nt = min(T, t1 - tb);
        if (lane == 0) mbar_arrive_expect_tx(bar, (uint32_t)(nt + (with_q ? 32 : 0)) * (uint32_t)W * 2u);
        __syncwarp();
        // q as mla_post_kernel left it: 16 rows of 16-bit heads, 16 rows of remainders (rows of heads that do not exist are zero)
        if (with_q) bulk_g2s(qh + (uint32_t)lane * LDB, qsplit + (size_t)lane * W, (uint32_t)W * 2u, bar);
        for (int j = lane; j < nt; j += 32) {
            const int t = tb + j, page = page_table[t / d.page_tokens], off = t % d.page_tokens;
            bulk_g2s(rows + (uint32_t)j * LDB, lat_pool + ((size_t)page * d.page_tokens + off) * W, (uint32_t)W * 2u, bar);
        }
    };
    if (warp == 0) fetch(t0, true);
    float acc[CW / 8][4];  // columns col0 + 8 nb + 2 (lane % 4) + {0, 1} of heads lane / 4 and lane / 4 + 8
#pragma unroll
    for (int nb = 0; nb < CW / 8; ++nb) acc[nb][0] = acc[nb][1] = acc[nb][2] = acc[nb][3] = 0.0f;
    const int g = lane >> 2, tq = lane & 3;
    uint32_t phase = 0;
    for (int tb = t0; tb < t1; tb += T) {
        const int nt = min(T, t1 - tb);
        // rows past the slice's end are multiplied by p = 0: they must hold finite values
        for (int i = tid; i < (T - nt) * (int)(LDB / 16); i += MLA_MMA_THREADS)
            *reinterpret_cast<uint4*>(rows_p + (size_t)(nt + i / (int)(LDB / 16)) * LDB + (size_t)(i % (int)(LDB / 16)) * 16) = make_uint4(0, 0, 0, 0);
        if (!mbar_wait(bar, phase)) atomicCAS(err, 0, DEV_ERR_FULL_WAIT);
        phase ^= 1u;
        __syncthreads();  // the zero rows are in place
        // ---- scores of positions 16 warp .. 16 warp + 15
        const int j0 = 16 * warp;
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
        if (j0 < nt) {
            const uint32_t a_off = (uint32_t)(lane & 15) * LDB + (uint32_t)(lane >> 4) * 16u;
            const uint32_t b_off = (uint32_t)(j0 + (lane & 7) + 8 * (lane >> 4)) * LDB + (uint32_t)((lane >> 3) & 1) * 16u;
#pragma unroll 4
            for (int ks = 0; ks < W / 16; ++ks) {
                uint32_t ah[4], al[4], b[4];
                ldsm_x4(ah, qh + a_off + (uint32_t)ks * 32u);
                ldsm_x4(al, ql + a_off + (uint32_t)ks * 32u);
                ldsm_x4(b, rows + b_off + (uint32_t)ks * 32u);
                Mma16<KT>::mma(c0, ah, b[0], b[1]);
                Mma16<KT>::mma(c0, al, b[0], b[1]);
                Mma16<KT>::mma(c1, ah, b[2], b[3]);
                Mma16<KT>::mma(c1, al, b[2], b[3]);
            }
        }
        {
            const int ja = j0 + 2 * tq, jb = j0 + 8 + 2 * tq;
            sc[g * LDS + ja] = c0[0] * scale;       sc[g * LDS + ja + 1] = c0[1] * scale;
            sc[(g + 8) * LDS + ja] = c0[2] * scale; sc[(g + 8) * LDS + ja + 1] = c0[3] * scale;
            sc[g * LDS + jb] = c1[0] * scale;       sc[g * LDS + jb + 1] = c1[1] * scale;
            sc[(g + 8) * LDS + jb] = c1[2] * scale; sc[(g + 8) * LDS + jb + 1] = c1[3] * scale;
        }
        __syncthreads();
        // ---- running softmax: eight threads per head, eight positions each
        {
            const int h = tid >> 3, sub = tid & 7;
            float v[8], mx = NEG;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int j = sub * 8 + i;
                v[i] = j < nt ? sc[h * LDS + j] : NEG;
                mx = fmaxf(mx, v[i]);
            }
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mold = mrun[h], mnew = fmaxf(mold, mx);
            float ps = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int j = sub * 8 + i;
                const float p = j < nt ? expf(v[i] - mnew) : 0.0f;
                ps += p;
                const KT hi = Elem<KT>::from_f32(p);
                ph[h * LDP + j] = hi;
                pl[h * LDP + j] = Elem<KT>::from_f32(p - Elem<KT>::to_f32(hi));
            }
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
            __syncwarp();
            if (sub == 0) {
                const float cr = expf(mold - mnew);
                corr[h] = cr;
                lrun[h] = lrun[h] * cr + ps;
                mrun[h] = mnew;
            }
        }
        __syncthreads();
        // ---- O += P V over this warp's latent columns
        {
            const float ca = corr[g], cb = corr[g + 8];
#pragma unroll
            for (int nb = 0; nb < CW / 8; ++nb) { acc[nb][0] *= ca; acc[nb][1] *= ca; acc[nb][2] *= cb; acc[nb][3] *= cb; }
            const uint32_t a_off = (uint32_t)(lane & 15) * (uint32_t)(LDP * 2) + (uint32_t)(lane >> 4) * 16u;
            const uint32_t v_off = (uint32_t)((lane & 7) + 8 * ((lane >> 3) & 1)) * LDB + (uint32_t)(col0 + 8 * (lane >> 4)) * 2u;
            for (int ks = 0; ks < T / 16; ++ks) {
                if (16 * ks >= nt) break;
                uint32_t ah[4], al[4];
                ldsm_x4(ah, pha + a_off + (uint32_t)ks * 32u);
                ldsm_x4(al, pla + a_off + (uint32_t)ks * 32u);
#pragma unroll
                for (int np = 0; np < CW / 16; ++np) {
                    if (col0 + 16 * np >= C) break;
                    uint32_t b[4];
                    ldsm_x4_trans(b, rows + v_off + (uint32_t)(16 * ks) * LDB + (uint32_t)np * 32u);
                    Mma16<KT>::mma(acc[2 * np], ah, b[0], b[1]);
                    Mma16<KT>::mma(acc[2 * np], al, b[0], b[1]);
                    Mma16<KT>::mma(acc[2 * np + 1], ah, b[2], b[3]);
                    Mma16<KT>::mma(acc[2 * np + 1], al, b[2], b[3]);
                }
            }
        }
        __syncthreads();  // every warp is done with the tile's rows
        if (warp == 0 && tb + T < t1) fetch(tb + T, false);
    }
#pragma unroll
    for (int nb = 0; nb < CW / 8; ++nb) {
        const int col = col0 + 8 * nb + 2 * tq;
        if (col >= C) break;
        float* pa = part_acc + ((size_t)s * d.heads + h0 + g) * C + col;
        if (g < H) *reinterpret_cast<float2*>(pa) = make_float2(acc[nb][0], acc[nb][1]);
        if (g + 8 < H) *reinterpret_cast<float2*>(pa + (size_t)8 * C) = make_float2(acc[nb][2], acc[nb][3]);
    }
    if (tid < H) {
        part_ml[((size_t)s * d.heads + h0 + tid) * 2 + 0] = mrun[tid];
        part_ml[((size_t)s * d.heads + h0 + tid) * 2 + 1] = lrun[tid];
    }
}

// ---------------------------------------------------------------------- routing rule
struct RouteRule {
    int experts, top;
    int groups, keep;  // experts form `groups` equal runs of neighbours; only the `keep` runs whose best score is largest may be chosen from
};
// One warp picks a token's experts: pr[experts] holds the router logits (shared memory, rewritten), gs[groups] is scratch.
// Scores are softmax(logits) over all experts; ties go to the lower index; each(k, expert, score)
// is called in every lane with the k-th choice and its score, unchanged.
template <class Each>
__device__ inline void route_pick(float* pr, float* gs, const RouteRule& r, int lane, Each each) {
    float mx = -INFINITY;
    for (int k = lane; k < r.experts; k += 32) mx = fmaxf(mx, pr[k]);
    mx = warp_max(mx);
    __syncwarp();
    for (int k = lane; k < r.experts; k += 32) pr[k] = expf(pr[k] - mx);
    __syncwarp();
    float sum = 0.0f;  // in expert order, the same in every lane
    for (int k = 0; k < r.experts; ++k) sum += pr[k];
    __syncwarp();
    for (int k = lane; k < r.experts; k += 32) pr[k] = pr[k] / sum;
    __syncwarp();
    auto best = [&](const float* v, int n, float& bv, int& bi) {
        bv = -INFINITY;
        bi = 0x7fffffff;
        for (int i = lane; i < n; i += 32) {
            const float t = v[i];
            if (t > bv || (t == bv && i < bi)) { bv = t; bi = i; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
        }
        if (bi >= n) bi = 0;  // nothing comparable (NaN logits): never an address past the list
    };
    float bv;
    int bi;
    if (r.keep < r.groups) {
        const int size = r.experts / r.groups;
        for (int g = lane; g < r.groups; g += 32) {
            float t = -INFINITY;
            for (int i = 0; i < size; ++i) t = fmaxf(t, pr[g * size + i]);
            gs[g] = t;
        }
        __syncwarp();
        for (int k = 0; k < r.keep; ++k) {
            best(gs, r.groups, bv, bi);
            __syncwarp();
            if (lane == 0) gs[bi] = -INFINITY;  // kept
            __syncwarp();
        }
        for (int i = lane; i < r.experts; i += 32)
            if (gs[i / size] != -INFINITY) pr[i] = -1.0f;  // scores are never negative: below any expert that may be chosen
        __syncwarp();
    }
    for (int k = 0; k < r.top; ++k) {
        best(pr, r.experts, bv, bi);
        each(k, bi, bv);
        __syncwarp();
        if (lane == 0) pr[bi] = -INFINITY;  // removed from the later rounds
        __syncwarp();
    }
}

// What the router multiplies: fill(xs) writes the vector to shared memory (all threads; the barriers of the block
// reductions publish it) and returns the factor its dot products still need; CTA 0 keeps the vector for the expert kernels.
struct RouterRmsIn {  // rmsnorm(x, gamma)
    const float *x, *gamma;
    float* out;
    __device__ float fill(float* xs, float* red, int dim, bool writer) const {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < dim; i += blockDim.x) {
            const float v = __ldcg(x + i);
            xs[i] = v * gamma[i];
            ss += v * v;
        }
        const float inv = 1.0f / sqrtf(block_sum(ss, red) * (1.0f / (float)dim) + RMS_EPS);
        if (writer)
            for (int i = threadIdx.x; i < dim; i += blockDim.x) out[i] = xs[i] * inv;
        return inv;
    }
};
struct RouterMixIn {  // the residual stream behind two parallel mixers (InParallelMix, mixers.cuh)
    const float *x, *yl, *yr, *wl, *wr, *gain;
    float* out;
    float mult, eps;
    int n;               // entries the norms are over (zeros behind them)
    __device__ float fill(float* xs, float* red, int dim, bool writer) const {  // dim is a multiple of 4
        const int n4 = dim / 4, step = blockDim.x;
        auto at = [](const float* p, int i) { return __ldcg(reinterpret_cast<const float4*>(p) + i); };
        auto weight = [](const float* p, int i) { return reinterpret_cast<const float4*>(p)[i]; };
        float4* x4 = reinterpret_cast<float4*>(xs);
        float sl = 0.0f, sr = 0.0f, ss = 0.0f;
#pragma unroll 4
        for (int i = threadIdx.x; i < n4; i += step) {
            const float4 a = at(yl, i), b = at(yr, i);
            sl += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
            sr += b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
        }
        const float rl = 0.5f / sqrtf(block_sum(sl, red) * (1.0f / (float)n) + eps);
        const float rr = 0.5f / sqrtf(block_sum(sr, red) * (1.0f / (float)n) + eps);
#pragma unroll 4
        for (int i = threadIdx.x; i < n4; i += step) {
            const float4 a = at(yl, i), b = at(yr, i), p = weight(wl, i), q = weight(wr, i);
            const float4 z = make_float4(a.x * rl * p.x + b.x * rr * q.x, a.y * rl * p.y + b.y * rr * q.y, a.z * rl * p.z + b.z * rr * q.z, a.w * rl * p.w + b.w * rr * q.w);
            x4[i] = z;
            ss += z.x * z.x + z.y * z.y + z.z * z.z + z.w * z.w;
        }
        const float r = mult / sqrtf(block_sum(ss, red) * (1.0f / (float)n) + eps);
#pragma unroll 4
        for (int i = threadIdx.x; i < n4; i += step) {
            const float4 b = at(x, i), g = weight(gain, i), z = x4[i];
            const float4 v = make_float4(b.x + z.x * r * g.x, b.y + z.y * r * g.y, b.z + z.z * r * g.z, b.w + z.w * r * g.w);
            x4[i] = v;
            if (writer) reinterpret_cast<float4*>(out)[i] = v;
        }
        __syncthreads();
        return 1.0f;
    }
};

// ---------------------------------------------------------------------- router: one warp per expert, the last CTA picks
// logit_e = W_r[e] . xn (every CTA forms xn, see above); the CTA that finishes last (a counter, nobody waits) applies the
// routing rule.  Besides the choice (sel_ids, sel_w) it writes the compact list of the chosen experts
// this rank holds (local index, weight, count): the expert kernels walk that list.
template <typename WT, class In>
__global__ void __launch_bounds__(128)
moe_router_kernel(In in, const WT* __restrict__ wr, float* __restrict__ logits, unsigned int* __restrict__ counter, int* __restrict__ sel_ids,
                  float* __restrict__ sel_w, int* __restrict__ loc_ids, float* __restrict__ loc_w, int* __restrict__ n_loc, int dim, RouteRule rule,
                  int e0, int n_local) {
    extern __shared__ __align__(16) float sm[];  // [dim] the input; the last CTA: [experts] scores and [groups] on top of it
    __shared__ float red[32];
    __shared__ int s_last;
    constexpr int EPC = Elem<WT>::EPC, PRE = 8;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const int n_experts = rule.experts;
    float* xg = sm;
    // this warp's expert row: its first chunks are requested before anything else (x, gamma and the row arrive together)
    const int e = min(blockIdx.x * nw + warp, n_experts - 1);
    const char* row = reinterpret_cast<const char*>(wr + (size_t)e * dim);
    const int nchunks = dim / EPC;
    uint4 w[PRE];
#pragma unroll
    for (int j = 0; j < PRE; ++j) w[j] = lane + 32 * j < nchunks ? ldg_stream(row + (size_t)(lane + 32 * j) * 16) : make_uint4(0, 0, 0, 0);
    pdl_wait();
    pdl_launch_dependents();  // after the wait: at most this kernel and the next one overlap
    const float inv = in.fill(xg, red, dim, blockIdx.x == 0);
    float a = 0.0f;
#pragma unroll
    for (int j = 0; j < PRE; ++j) {
        const int c = lane + 32 * j;
        if (c < nchunks) {
            float f[EPC];
            Elem<WT>::unpack(w[j], f);
#pragma unroll
            for (int k = 0; k < EPC; ++k) a = fmaf(f[k], xg[c * EPC + k], a);
        }
    }
    for (int c = lane + 32 * PRE; c < nchunks; c += 32) {
        float f[EPC];
        Elem<WT>::unpack(ldg_stream(row + (size_t)c * 16), f);
#pragma unroll
        for (int k = 0; k < EPC; ++k) a = fmaf(f[k], xg[c * EPC + k], a);
    }
    a = warp_sum(a) * inv;
    if (lane == 0 && blockIdx.x * nw + warp < n_experts) logits[e] = a;
    __threadfence();
    __syncthreads();
    if (tid == 0) s_last = atomicAdd(counter, 1u) == gridDim.x - 1 ? 1 : 0;
    __syncthreads();
    if (!s_last || warp != 0) return;
    __threadfence();
    float* pr = sm;  // the input is no longer needed: the other warps have left, this one has its logit
    for (int k = lane; k < n_experts; k += 32) pr[k] = __ldcg(logits + k);
    __syncwarp();
    int nl = 0;
    route_pick(pr, pr + n_experts, rule, lane, [&](int k, int bi, float bv) {
        const bool here = bi >= e0 && bi < e0 + n_local;
        if (lane == 0) {
            sel_ids[k] = bi;
            sel_w[k] = bv;
            if (here) { loc_ids[nl] = bi - e0; loc_w[nl] = bv; }
        }
        if (here) ++nl;  // bi is the same in every lane
    });
    if (lane == 0) {
        *n_loc = nl;
        *counter = 0u;  // for the next launch
    }
}

struct MoeDims {
    int dim, hidden;
    int shared_cols;      // columns of the shared FFN this rank holds
};
// the chosen experts this rank holds, in the router's order: local index, weight; their count
struct MoePick {
    const int* loc_ids;
    const float* loc_w;
    const int* n_loc;
};

// ---------------------------------------------------------------------- gate = silu(xn W1) * (xn W3) * weight
// Units: for each chosen local expert `hidden` column pairs, then `shared_cols` pairs of the shared FFN; one
// warp per unit (rows 2j and 2j + 1 of an interleaved [2 hidden, dim] matrix are adjacent in memory).
// This and moe_w2_kernel are the plain-load forms, for shapes the streamed GEMV does not take.
template <typename WT>
__global__ void __launch_bounds__(256)
moe_w13_kernel(const float* __restrict__ xn, const WT* __restrict__ w13, const WT* __restrict__ ws13, MoePick pick,
               float* __restrict__ gate, MoeDims d) {
    extern __shared__ float xs[];  // [dim]
    const int tid = threadIdx.x, lane = tid & 31;
    pdl_wait();
    pdl_launch_dependents();  // after the wait: at most this kernel and the next one overlap
    for (int i = tid; i < d.dim; i += blockDim.x) xs[i] = __ldcg(xn + i);
    __syncthreads();
    const int nl = __ldcg(pick.n_loc);
    const int units = nl * d.hidden + d.shared_cols;
    const int gw = (blockIdx.x * blockDim.x + tid) >> 5, total = (gridDim.x * blockDim.x) >> 5;
    for (int u = gw; u < units; u += total) {
        const WT* rows;
        float weight = 1.0f;
        if (u < nl * d.hidden) {
            const int s = u / d.hidden, j = u % d.hidden;
            rows = w13 + ((size_t)__ldcg(pick.loc_ids + s) * d.hidden + j) * 2 * d.dim;
            weight = __ldcg(pick.loc_w + s);
        } else {
            rows = ws13 + (size_t)(u - nl * d.hidden) * 2 * d.dim;
        }
        float y[2];
        warp_rows_dot<WT, 2>(rows, (size_t)d.dim, xs, d.dim, lane, y);
        if (lane == 0) gate[u] = (y[0] / (1.0f + expf(-y[0]))) * y[1] * weight;
    }
}

// ---------------------------------------------------------------------- y = sum of W2 gate over the local experts and the shared FFN
// One warp per output row.  Single GPU: out = res + alpha y.  Expert parallel: y goes to every rank's inbox
// (the dense model's push all-reduce, TpRegion); the next GEMV's prologue adds the ranks' rows in rank order.
template <typename WT>
__global__ void __launch_bounds__(256)
moe_w2_kernel(const float* __restrict__ gate, const WT* __restrict__ w2, const WT* __restrict__ ws2, MoePick pick,
              const float* __restrict__ res, float* __restrict__ out, float alpha, MoeDims d, TpLink tp) {
    extern __shared__ float gs[];  // [n_loc * hidden + shared_cols]
    const int tid = threadIdx.x, lane = tid & 31;
    pdl_wait();
    pdl_launch_dependents();  // after the wait: at most this kernel and the next one overlap
    const int nl = __ldcg(pick.n_loc);
    const int units = nl * d.hidden + d.shared_cols;
    for (int i = tid; i < units; i += blockDim.x) gs[i] = __ldcg(gate + i);
    __syncthreads();
    const int gw = (blockIdx.x * blockDim.x + tid) >> 5, total = (gridDim.x * blockDim.x) >> 5;
    constexpr int EPC = Elem<WT>::EPC;
    for (int r = gw; r < d.dim; r += total) {
        float a = 0.0f;  // this lane's share of the row's sum over every segment: one reduction at the end, loads of all segments independent
        for (int s = 0; s <= nl; ++s) {
            const WT* seg;
            const float* g = gs + s * d.hidden;
            int K;
            if (s < nl) {
                seg = w2 + ((size_t)__ldcg(pick.loc_ids + s) * d.dim + r) * d.hidden; K = d.hidden;
            } else {
                if (d.shared_cols == 0) continue;
                seg = ws2 + (size_t)r * d.shared_cols; K = d.shared_cols;
            }
#pragma unroll 4
            for (int c = lane; c < K / EPC; c += 32) {
                const uint4 w = ldg_stream(reinterpret_cast<const char*>(seg) + (size_t)c * 16);
                float f[EPC];
                Elem<WT>::unpack(w, f);
#pragma unroll
                for (int e = 0; e < EPC; e += 4) {
                    const float4 x4 = *reinterpret_cast<const float4*>(g + c * EPC + e);
                    a = fmaf(f[e], x4.x, a); a = fmaf(f[e + 1], x4.y, a); a = fmaf(f[e + 2], x4.z, a); a = fmaf(f[e + 3], x4.w, a);
                }
            }
        }
        const float y = warp_sum(a);
        if (lane == 0) {
            if (tp.world > 1) {
                const unsigned int seq = __ldcg(&tp.st->ar_base) + (unsigned int)tp.ar_out;
                const size_t at = ((size_t)(seq % 3u) * tp.world + tp.rank) * tp.dim + r;
                const float v = tp_sanitize(y);
                for (int p = 0; p < tp.world; ++p) reinterpret_cast<float*>(tp.peers[p])[at] = v;
            } else {
                out[r] = __ldcg(res + r) + alpha * y;
            }
        }
    }
}

}  // namespace cd
