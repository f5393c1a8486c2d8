// The configured decoder's mixers, routing and vector steps over many prompt tokens at once (tensor cores: mma.sync for
// the mixers, whose operands are produced in the kernel; the linears are pf_gemm_kernel, prefill.cuh).  Same
// arithmetic as the one-token kernels of mixers.cuh; fp32 operands enter the tensor cores as a 16-bit value and a 16-bit
// remainder, so a product keeps 16 (bf16) or 22 (fp16) mantissa bits.
#pragma once
#include "mixers.cuh"
#include "moe.cuh"
#include "prefill.cuh"

namespace cd {

constexpr int MEM_CHUNK = 64;     // prompt tokens per chunk of the matrix memory
constexpr int MEM_LD = 72;        // row stride of a 64-wide bf16 tile in shared memory (ldmatrix without bank conflicts)

template <typename T> __device__ inline uint32_t pack2(float a, float b) {
    const T x = Elem<T>::from_f32(a), y = Elem<T>::from_f32(b);
    return (uint32_t)*reinterpret_cast<const unsigned short*>(&x) | (uint32_t)*reinterpret_cast<const unsigned short*>(&y) << 16;
}
template <typename T> __device__ inline float round16(float v) { return Elem<T>::to_f32(Elem<T>::from_f32(v)); }

// ---------------------------------------------------------------------- after the projections: q, k and v of the attention
// One CTA per token: whole-projection norms or rotation, temperature on q; q as 16-bit head and remainder
// [rows][H * maps * kp], the key and value rows into their pages.
template <typename KT>
__global__ void __launch_bounds__(256) attn_rows_kernel(const float* __restrict__ proj, int ld, AttnDims a, ProjLayout pl, const float* __restrict__ q_norm,
                                                        const float* __restrict__ k_norm, const int* __restrict__ page_table, KT* __restrict__ pool,
                                                        KT* __restrict__ q_hi, KT* __restrict__ q_lo, int pos0) {
    __shared__ float red[32];
    const float* row = proj + (size_t)blockIdx.x * ld;
    const int pos = pos0 + blockIdx.x, tid = threadIdx.x, nq = a.H * a.maps * a.dim, nk = a.G * a.maps * a.dim;
    float rq = a.temperature(pos), rk = 1.0f;
    if (q_norm != nullptr) {
        float sq = 0.0f, sk = 0.0f;
        for (int i = tid; i < nq; i += 256) sq = fmaf(row[pl.lq + i], row[pl.lq + i], sq);
        for (int i = tid; i < nk; i += 256) sk = fmaf(row[pl.lk + i], row[pl.lk + i], sk);
        rq /= sqrtf(block_sum(sq, red) / (float)nq + a.eps);
        rk = 1.0f / sqrtf(block_sum(sk, red) / (float)nk + a.eps);
    }
    __shared__ float2 cs_sm[128];  // dims is at most 256
    a.rot.fill(cs_sm, pos);
    __syncthreads();
    // two neighbouring entries (a rotated pair) of a [head][map][kp] vector
    auto pair = [&](const float* src, const float* norm, int i, float r, float& u, float& v) {
        const int hm = i / a.kp, d = i % a.kp;
        const float* p = src + hm * a.dim;
        u = d < a.dim ? p[d] * r * (norm != nullptr ? norm[hm * a.dim + d] : 1.0f) : 0.0f;
        v = d + 1 < a.dim ? p[d + 1] * r * (norm != nullptr ? norm[hm * a.dim + d + 1] : 1.0f) : 0.0f;
        if (d < a.rot.dims) {
            const float2 cs = cs_sm[d >> 1];
            const float t = u * cs.x - v * cs.y;
            v = v * cs.x + u * cs.y;
            u = t;
        }
    };
    float u, v;
    for (int i = 2 * tid; i < a.H * a.kr(); i += 512) {
        pair(row + pl.lq, q_norm, i, rq, u, v);
        pf_store(q_hi, q_lo, (size_t)blockIdx.x * a.H * a.kr() + i, u);
        pf_store(q_hi, q_lo, (size_t)blockIdx.x * a.H * a.kr() + i + 1, v);
    }
    const int page = page_table[pos / a.page_tokens], off = pos % a.page_tokens;
    for (int i = 2 * tid; i < a.G * a.kr(); i += 512) {
        pair(row + pl.lk, k_norm, i, rk, u, v);
        KT* k = pool + a.k_at(page, i / a.kr(), off) + i % a.kr();
        k[0] = Elem<KT>::from_f32(u);
        k[1] = Elem<KT>::from_f32(v);
    }
    for (int i = tid; i < a.G * a.vp; i += 256) {
        const int g = i / a.vp, d = i % a.vp;
        pool[a.v_at(page, g, off) + d] = Elem<KT>::from_f32(d < a.vdim ? row[pl.lv + g * a.vdim + d] : 0.0f);
    }
}

// ---------------------------------------------------------------------- windowed attention of the prompt
// grid = (ceil(rows / 64), heads * maps), four warps of 16 query rows.  Visible keys are walked 64 at a time straight out
// of the pages (cp.async, two tiles in flight), scores and the running softmax stay in registers.
constexpr int AW_TILE = 64;
__host__ __device__ inline size_t attn_window_smem(int kp, int vp) { return (size_t)AW_TILE * (4 * (kp + 8) + 2 * (vp + 8)) * 2; }

__device__ inline void cp_async16(uint32_t dst, const void* src, uint32_t bytes) {  // bytes 16 or 0 (zero fill)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ inline void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ inline void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

struct AttnWindow {
    AttnDims a;
    const float* slopes;   // nullptr: no distance bias
    const float* sink;     // nullptr: none
    const float* proj;     // gate projections: row ld, column gate_off + head (a gate per head is applied here)
    int proj_ld, gate_off;
    const int* page_table;
    int rows, pos0;        // query rows and the position of the first
    int out_ld;            // row stride of the output [rows][H * vdim], padded with zeros
    float* raw;            // not nullptr: the maps' outputs [rows][H * maps][vdim] go here instead, in fp32
};

template <typename KT, typename AT, int VD>
__global__ void __launch_bounds__(128) attn_window_kernel(const __grid_constant__ AttnWindow p, const KT* __restrict__ q_hi, const KT* __restrict__ q_lo,
                                                          const KT* __restrict__ pool, AT* __restrict__ out_hi, AT* __restrict__ out_lo) {
    extern __shared__ __align__(128) unsigned char aw_raw[];
    constexpr float NEG = -3.402823466e+38f;
    const AttnDims& a = p.a;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, hm = blockIdx.y, h = hm / a.maps, g = h / (a.H / a.G);
    const int r0 = blockIdx.x * AW_TILE, map_off = (hm % a.maps) * a.kp;
    const uint32_t ldk = (uint32_t)(a.kp + 8) * 2u, ldv = (uint32_t)(a.vp + 8) * 2u;
    const uint32_t qh = smem_addr(aw_raw), ql = qh + AW_TILE * ldk, ks0 = ql + AW_TILE * ldk, vs0 = ks0 + 2 * AW_TILE * ldk;
    const int p_first = p.pos0 + r0, p_last = min(p.pos0 + p.rows, p.pos0 + r0 + AW_TILE) - 1;
    const int lo = a.window > 0 ? max(0, p_first - a.window + 1) : 0;
    const int ntiles = (p_last - lo) / AW_TILE + 1;
    const int kch = a.kp / 8, vch = a.vp / 8;
    for (int i = tid; i < AW_TILE * kch; i += 128) {
        const int r = i / kch, c = i % kch;
        const bool ok = r0 + r < p.rows;
        const size_t at = ((size_t)(ok ? r0 + r : 0) * a.H * a.maps + hm) * a.kp + c * 8;
        cp_async16(qh + r * ldk + c * 16, q_hi + at, ok ? 16 : 0);
        cp_async16(ql + r * ldk + c * 16, q_lo + at, ok ? 16 : 0);
    }
    auto fetch = [&](int tile) {
        const uint32_t kd = ks0 + (tile & 1) * AW_TILE * ldk, vd = vs0 + (tile & 1) * AW_TILE * ldv;
        for (int i = tid; i < AW_TILE * kch; i += 128) {
            const int r = i / kch, c = i % kch, t = lo + tile * AW_TILE + r;
            const bool ok = t <= p_last;
            const int tt = ok ? t : p_last;
            cp_async16(kd + r * ldk + c * 16, pool + a.k_at(p.page_table[tt / a.page_tokens], g, tt % a.page_tokens) + map_off + c * 8, ok ? 16 : 0);
        }
        for (int i = tid; i < AW_TILE * vch; i += 128) {
            const int r = i / vch, c = i % vch, t = lo + tile * AW_TILE + r;
            const bool ok = t <= p_last;
            const int tt = ok ? t : p_last;
            cp_async16(vd + r * ldv + c * 16, pool + a.v_at(p.page_table[tt / a.page_tokens], g, tt % a.page_tokens) + c * 8, ok ? 16 : 0);
        }
        cp_async_commit();
    };
    fetch(0);
    const int gq = lane >> 2, tq = lane & 3;
    const int row_a = r0 + 16 * warp + gq, row_b = row_a + 8;  // this lane's two query rows
    const int pa = p.pos0 + row_a, pb = p.pos0 + row_b;
    const float slope = p.slopes != nullptr ? p.slopes[h] : 0.0f;
    float m_a = NEG, m_b = NEG, l_a = 0.0f, l_b = 0.0f;
    float o[VD / 8][4];
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const uint32_t a_off = (uint32_t)(16 * warp + (lane & 15)) * ldk + (uint32_t)(lane >> 4) * 16u;
    const uint32_t b_off = (uint32_t)((lane & 7) + 8 * (lane >> 4)) * ldk + (uint32_t)((lane >> 3) & 1) * 16u;
    const uint32_t v_off = (uint32_t)((lane & 7) + 8 * ((lane >> 3) & 1)) * ldv + (uint32_t)(8 * (lane >> 4)) * 2u;
    for (int tile = 0; tile < ntiles; ++tile) {
        if (tile + 1 < ntiles) {
            fetch(tile + 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t kt = ks0 + (tile & 1) * AW_TILE * ldk, vt = vs0 + (tile & 1) * AW_TILE * ldv;
        float s[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        for (int k = 0; k < a.kp / 16; ++k) {
            uint32_t ah[4], al[4];
            ldsm_x4(ah, qh + a_off + (uint32_t)k * 32u);
            ldsm_x4(al, ql + a_off + (uint32_t)k * 32u);
            uint32_t b[4][4];
#pragma unroll
            for (int n = 0; n < 4; ++n) ldsm_x4(b[n], kt + b_off + (uint32_t)(16 * n) * ldk + (uint32_t)k * 32u);
            // the two products of an accumulator are kept apart: back to back the second would wait for the first
#pragma unroll
            for (int n = 0; n < 4; ++n) { Mma16<KT>::mma(s[2 * n], ah, b[n][0], b[n][1]); Mma16<KT>::mma(s[2 * n + 1], ah, b[n][2], b[n][3]); }
#pragma unroll
            for (int n = 0; n < 4; ++n) { Mma16<KT>::mma(s[2 * n], al, b[n][0], b[n][1]); Mma16<KT>::mma(s[2 * n + 1], al, b[n][2], b[n][3]); }
        }
        const int j0 = lo + tile * AW_TILE + 2 * tq;
        float x_a = NEG, x_b = NEG;
        auto score = [&](float v, int i, int j) {  // NEG: out of sight
            const int d = i - j;
            return d >= 0 && (a.window <= 0 || d < a.window) ? v * a.scale - slope * (float)d : NEG;
        };
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            const int j = j0 + 8 * n;
            s[n][0] = score(s[n][0], pa, j); s[n][1] = score(s[n][1], pa, j + 1);
            s[n][2] = score(s[n][2], pb, j); s[n][3] = score(s[n][3], pb, j + 1);
            x_a = fmaxf(x_a, fmaxf(s[n][0], s[n][1]));
            x_b = fmaxf(x_b, fmaxf(s[n][2], s[n][3]));
        }
#pragma unroll
        for (int w = 1; w < 4; w <<= 1) {
            x_a = fmaxf(x_a, __shfl_xor_sync(0xffffffffu, x_a, w));
            x_b = fmaxf(x_b, __shfl_xor_sync(0xffffffffu, x_b, w));
        }
        const float n_a = fmaxf(m_a, x_a), n_b = fmaxf(m_b, x_b);
        const float c_a = expf(m_a - n_a), c_b = expf(m_b - n_b);
        m_a = n_a; m_b = n_b;
        l_a *= c_a; l_b *= c_b;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            s[n][0] = s[n][0] > NEG ? expf(s[n][0] - m_a) : 0.0f; s[n][1] = s[n][1] > NEG ? expf(s[n][1] - m_a) : 0.0f;
            s[n][2] = s[n][2] > NEG ? expf(s[n][2] - m_b) : 0.0f; s[n][3] = s[n][3] > NEG ? expf(s[n][3] - m_b) : 0.0f;
            l_a += s[n][0] + s[n][1];
            l_b += s[n][2] + s[n][3];
        }
#pragma unroll
        for (int i = 0; i < VD / 8; ++i) { o[i][0] *= c_a; o[i][1] *= c_a; o[i][2] *= c_b; o[i][3] *= c_b; }
#pragma unroll
        for (int k = 0; k < 4; ++k) {  // 16 keys at a time: the score fragments are the probability operand's fragments
            const float* s0 = s[2 * k];
            const float* s1 = s[2 * k + 1];
            const uint32_t ph[4] = {pack2<KT>(s0[0], s0[1]), pack2<KT>(s0[2], s0[3]), pack2<KT>(s1[0], s1[1]), pack2<KT>(s1[2], s1[3])};
            const uint32_t pl[4] = {pack2<KT>(s0[0] - round16<KT>(s0[0]), s0[1] - round16<KT>(s0[1])), pack2<KT>(s0[2] - round16<KT>(s0[2]), s0[3] - round16<KT>(s0[3])),
                                    pack2<KT>(s1[0] - round16<KT>(s1[0]), s1[1] - round16<KT>(s1[1])), pack2<KT>(s1[2] - round16<KT>(s1[2]), s1[3] - round16<KT>(s1[3]))};
#pragma unroll
            for (int n = 0; n < VD / 16; n += 2) {
                if (16 * n < a.vp) {
                    const bool two = 16 * (n + 1) < a.vp;
                    uint32_t b[4], c[4];
                    ldsm_x4_trans(b, vt + v_off + (uint32_t)(16 * k) * ldv + (uint32_t)n * 32u);
                    if (two) ldsm_x4_trans(c, vt + v_off + (uint32_t)(16 * k) * ldv + (uint32_t)(n + 1) * 32u);
                    else c[0] = c[1] = c[2] = c[3] = 0u;
                    Mma16<KT>::mma(o[2 * n], ph, b[0], b[1]);
                    Mma16<KT>::mma(o[2 * n + 1], ph, b[2], b[3]);
                    Mma16<KT>::mma(o[2 * n + 2], ph, c[0], c[1]);
                    Mma16<KT>::mma(o[2 * n + 3], ph, c[2], c[3]);
                    Mma16<KT>::mma(o[2 * n], pl, b[0], b[1]);
                    Mma16<KT>::mma(o[2 * n + 1], pl, b[2], b[3]);
                    Mma16<KT>::mma(o[2 * n + 2], pl, c[0], c[1]);
                    Mma16<KT>::mma(o[2 * n + 3], pl, c[2], c[3]);
                }
            }
        }
        __syncthreads();  // the tile's buffers may be refilled
    }
#pragma unroll
    for (int w = 1; w < 4; w <<= 1) {
        l_a += __shfl_xor_sync(0xffffffffu, l_a, w);
        l_b += __shfl_xor_sync(0xffffffffu, l_b, w);
    }
    const float sink = p.sink != nullptr ? p.sink[h] : NEG;
    auto finish = [&](int row, float m, float l) {  // factor of the row's accumulators: sink in the denominator, head gate
        if (row >= p.rows) return 0.0f;
        const float M = fmaxf(m, sink), e = expf(m - M);
        const float f = e / (l * e + (p.sink != nullptr ? expf(sink - M) : 0.0f));
        return a.gate == 1 ? f * sigmoid(p.proj[(size_t)row * p.proj_ld + p.gate_off + h]) : f;
    };
    const float f_a = finish(row_a, m_a, l_a), f_b = finish(row_b, m_b, l_b);
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) {
        const int c = 8 * n + 2 * tq;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            if (c + e < a.vdim) {
                if (p.raw != nullptr) {
                    if (row_a < p.rows) p.raw[((size_t)row_a * a.H * a.maps + hm) * a.vdim + c + e] = o[n][e] * f_a;
                    if (row_b < p.rows) p.raw[((size_t)row_b * a.H * a.maps + hm) * a.vdim + c + e] = o[n][2 + e] * f_b;
                } else {
                    if (row_a < p.rows) pf_store(out_hi, out_lo, (size_t)row_a * p.out_ld + h * a.vdim + c + e, o[n][e] * f_a);
                    if (row_b < p.rows) pf_store(out_hi, out_lo, (size_t)row_b * p.out_ld + h * a.vdim + c + e, o[n][2 + e] * f_b);
                }
            }
        }
    }
    if (p.raw != nullptr) return;
    if (h == a.H - 1)
        for (int r = tid; r < AW_TILE && r0 + r < p.rows; r += 128)
            for (int c = a.H * a.vdim; c < p.out_ld; ++c) pf_store(out_hi, out_lo, (size_t)(r0 + r) * p.out_ld + c, 0.0f);
}

// per token: the second map's output subtracted from the first's, each head divided by its root mean square, times the
// constant factor and the gate of every element; one warp per head
template <typename AT>
__global__ void __launch_bounds__(256) diff_rows_kernel(const float* __restrict__ raw, const float* __restrict__ proj, int proj_ld, int gate_off, AttnDims a,
                                                        AT* __restrict__ hi, AT* __restrict__ lo, int ld) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float* gate = proj + (size_t)blockIdx.x * proj_ld + gate_off;
    for (int h = warp; h < a.H; h += 8) {
        const float* o1 = raw + ((size_t)blockIdx.x * a.H + h) * 2 * a.vdim;
        const float* o2 = o1 + a.vdim;
        float ss = 0.0f;
        for (int i = lane; i < a.vdim; i += 32) { const float v = o1[i] - a.lambda * o2[i]; ss = fmaf(v, v, ss); }
        const float r = a.out_scale / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
        for (int i = lane; i < a.vdim; i += 32) {
            const int j = h * a.vdim + i;
            pf_store(hi, lo, (size_t)blockIdx.x * ld + j, (o1[i] - a.lambda * o2[i]) * r * (a.gate == 2 ? sigmoid(gate[j]) : a.gate == 1 ? sigmoid(gate[h]) : 1.0f));
        }
    }
    for (int j = a.H * a.vdim + threadIdx.x; j < ld; j += 256) pf_store(hi, lo, (size_t)blockIdx.x * ld + j, 0.0f);
}

// ---------------------------------------------------------------------- latent attention of the prompt
// Keys and values of the visible positions are expanded once per piece into a buffer laid out like one page, then attended
// to by attn_window_kernel.  latent_rows_kernel: one CTA per new token, q as 16-bit head and remainder [rows][H][kp], the
// cache row [normed latent | rotated key].
template <typename KT>
__global__ void __launch_bounds__(256) latent_rows_kernel(const float* __restrict__ proj, int ld, MlaDims d, Rotation rot, const float* __restrict__ gamma,
                                                          const int* __restrict__ page_table, KT* __restrict__ pool, KT* __restrict__ q_hi, KT* __restrict__ q_lo,
                                                          int kp, int pos0) {
    __shared__ float red[32];
    const float* row = proj + (size_t)blockIdx.x * ld;
    const int pos = pos0 + blockIdx.x, tid = threadIdx.x, QH = d.nope_n + d.rope_n;
    __shared__ float2 cs_sm[128];  // nope + rope is at most 256
    auto cs_of = [&](int k) { return cs_sm[k]; };
    rot.fill(cs_sm, pos);
    __syncthreads();
    for (int i = tid; i < d.heads * kp; i += 256) {
        const int h = i / kp, k = i % kp;
        const float* q = row + h * QH;
        const float v = k < d.nope_n ? q[k] : k < QH ? rot.entry(k - d.nope_n, cs_of, [&](int j) { return q[d.nope_n + j]; }) : 0.0f;
        pf_store(q_hi, q_lo, (size_t)blockIdx.x * d.heads * kp + i, v);
    }
    const float* craw = row + d.heads * QH;
    float ss = 0.0f;
    for (int i = tid; i < d.latent_n; i += 256) ss = fmaf(craw[i], craw[i], ss);
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)d.latent_n + d.eps);
    KT* out = pool + ((size_t)page_table[pos / d.page_tokens] * d.page_tokens + pos % d.page_tokens) * d.row();
    for (int i = tid; i < d.latent; i += 256) out[i] = Elem<KT>::from_f32(i < d.latent_n ? craw[i] * r * gamma[i] : 0.0f);
    for (int i = tid; i < d.rope; i += 256) out[d.latent + i] = Elem<KT>::from_f32(i < d.rope_n ? rot.entry(i, cs_of, [&](int j) { return craw[d.latent_n + j]; }) : 0.0f);
}

// cached rows base, base + 1, ..: the latent as a GEMM operand [n][latent], the rotated key behind every head's expanded one
// (`x` describes the expanded buffer), zeros in its padding.  One CTA per position.
template <typename KT, typename AT>
__global__ void __launch_bounds__(256) latent_gather_kernel(const KT* __restrict__ pool, const int* __restrict__ page_table, MlaDims d, int base, AT* __restrict__ hi,
                                                            AT* __restrict__ lo, KT* __restrict__ expanded, AttnDims x) {
    const int pos = base + blockIdx.x, tid = threadIdx.x;
    const KT* row = pool + ((size_t)page_table[pos / d.page_tokens] * d.page_tokens + pos % d.page_tokens) * d.row();
    for (int i = tid; i < d.latent; i += 256) pf_store(hi, lo, (size_t)blockIdx.x * d.latent + i, Elem<KT>::to_f32(row[i]));
    const int nk = x.kp - d.nope_n, nv = x.vp - x.vdim;
    const KT zero = Elem<KT>::from_f32(0.0f);
    for (int i = tid; i < x.H * nk; i += 256) {
        const int h = i / nk, k = i % nk;
        expanded[x.k_at(0, h, blockIdx.x) + d.nope_n + k] = k < d.rope_n ? row[d.latent + k] : zero;
    }
    for (int i = tid; i < x.H * nv; i += 256) expanded[x.v_at(0, i / nv, blockIdx.x) + x.vdim + i % nv] = zero;
}

// output columns [H][nope] keys, then [H][vdim] values, of the expansion GEMM
template <typename KT> struct PfEpiExpand {
    KT* expanded;
    AttnDims x;
    int nope;
    __device__ void operator()(int, int row, int col, const float (&v)[32]) const {
        const int keys = x.H * nope;
        int h = col < keys ? col / nope : (col - keys) / x.vdim, d = col < keys ? col % nope : (col - keys) % x.vdim;
        bool key = col < keys;
        if (h >= x.H) return;
        KT* dst = expanded + (key ? x.k_at(0, h, row) : x.v_at(0, h, row));
        if (nope % 32 == 0 && x.vdim % 32 == 0) {  // the 32 columns are one head's, and so aligned
#pragma unroll
            for (int i = 0; i < 4; ++i)
                *reinterpret_cast<uint4*>(dst + d + 8 * i) = make_uint4(pack2<KT>(v[8 * i], v[8 * i + 1]), pack2<KT>(v[8 * i + 2], v[8 * i + 3]),
                                                                        pack2<KT>(v[8 * i + 4], v[8 * i + 5]), pack2<KT>(v[8 * i + 6], v[8 * i + 7]));
            return;
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) {
            dst[d] = Elem<KT>::from_f32(v[i]);
            if (++d == (key ? nope : x.vdim)) {
                d = 0;
                if (++h == x.H) {
                    if (!key) return;  // columns past the last value
                    key = false;
                    h = 0;
                }
                dst = expanded + (key ? x.k_at(0, h, row) : x.v_at(0, h, row));
            }
        }
    }
};

// ---------------------------------------------------------------------- token side: gate of the second embedding's part
template <typename AT, typename WT> struct PfEpiTokenGate {
    AT *hi, *lo;
    int ld;               // columns of the operand, zeros behind `dim`
    const WT* table;      // the layer's first column
    int table_ld, dim;
    const uint32_t* ids;
    __device__ void operator()(int, int row, int col, const float (&v)[32]) const {
        const WT* e = table + (size_t)ids[row] * table_ld;
        float g[32];
        const bool run = col + 32 <= dim && table_ld % 8 == 0 && (reinterpret_cast<size_t>(table) & 15) == 0;
        if (run) {
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
                float f[8];
                Elem<WT>::unpack(ldg_stream(e + col + i), f);
#pragma unroll
                for (int k = 0; k < 8; ++k) g[i + k] = f[k];
            }
        } else {  // every entry is requested before anything is stored
#pragma unroll
            for (int i = 0; i < 32; ++i) g[i] = col + i < dim ? Elem<WT>::to_f32(__ldg(e + col + i)) : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) g[i] *= gelu_tanh(v[i]);
        if (run) {  // (dim >= col + 32, so the operand's rows hold them)
            pf_store_run(hi, lo, (size_t)row * ld + col, g);
        } else {
#pragma unroll
            for (int i = 0; i < 32; ++i)
                if (col + i < ld) pf_store(hi, lo, (size_t)row * ld + col + i, g[i]);
        }
    }
};

// ---------------------------------------------------------------------- matrix memory of the prompt, chunk by chunk
// With F_t the running sum of the log forget gates inside a chunk and a_s = i_s - F_s, the recurrence unrolls to
//   M_t = max(m_0, max_{s <= t} a_s),  m_t = F_t + M_t,
//   S_t^T q = e^{m_0 - M_t} S_0^T q + sum_{s <= t} e^{a_s - M_t} (k_s . q) v_s     (n . q likewise),
// so a chunk needs only the state it starts from.  Three kernels: every chunk's own contribution to the state, a scan over
// the chunks that turns the contributions into starting states, and the read-outs of all chunks.
// Linear attention is the case with log forget gate ln(decay), input gate 1 and no maximum or normaliser: F_t = (t + 1) ln
// decay, every scale e^0, and M_t = -F_t in the read-out; its q, k and v arrive activated.
struct MemPrompt {
    MemDims d;
    ProjLayout pl;
    const float* proj;
    int proj_ld;
    const float *ib, *fb;
    int rows, nchunk;
    float* state;        // the layer's live state: read at the start, rewritten with the state behind the last row
    float* U;            // [nchunk][H][dim][vs]  contributions, then starting states
    float* UN;           // [nchunk][H][dim]      the same of n
    float* gm;           // [nchunk][H][2]        sum of the log forget gates, largest log weight; then [1] = starting maximum
    float* m_live;       // [H] the live maximum at the start
    float* out;          // [rows][H * vdim]
};

// gates of one chunk: F (inclusive running sum of log forget gates) and I (log input gates) of 64 tokens; tokens past the
// end forget nothing and add nothing.  Ends with a barrier.
__device__ inline void mem_chunk_gates(const MemPrompt& p, int h, int t0, int nt, float* F, float* I, float* tmp) {
    const int tid = threadIdx.x;
    if (p.d.linear()) {
        if (tid < MEM_CHUNK) {
            F[tid] = (float)min(tid + 1, nt) * p.d.log_decay[h];
            I[tid] = tid < nt ? 0.0f : -INFINITY;
        }
        __syncthreads();
        return;
    }
    if (tid < MEM_CHUNK) {
        float gi = -INFINITY, gf = 0.0f;
        if (tid < nt) {
            const float* row = p.proj + (size_t)(t0 + tid) * p.proj_ld;
            gi = soft_cap(row[p.pl.ri + h] + p.ib[h], p.d.cap);
            gf = log_sigmoid(soft_cap(row[p.pl.rf + h] + p.fb[h], p.d.cap));
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, gf, o);
            if ((tid & 31) >= o) gf += v;
        }
        if (tid == 31) *tmp = gf;
        F[tid] = gf;
        I[tid] = gi;
    }
    __syncthreads();
    if (tid >= 32 && tid < MEM_CHUNK) F[tid] += *tmp;
    __syncthreads();
}

// a [64][64] tile of fp32 rows as bf16 head and remainder; rows >= nrows and columns >= ncols are zero; row_scale may be null
__device__ inline void mem_load_tile(__nv_bfloat16* hi, __nv_bfloat16* lo, const float* src, size_t ld, int nrows, int ncols, const float* row_scale, float scale) {
#pragma unroll 8
    for (int i = threadIdx.x; i < 64 * 64; i += 128) {
        const int r = i >> 6, c = i & 63;
        float v = 0.0f;
        if (r < nrows && c < ncols) v = src[(size_t)r * ld + c] * (row_scale ? row_scale[r] : scale);
        pf_store(hi, lo, (size_t)r * MEM_LD + c, v);
    }
}
constexpr int MEM_TILE_ELEMS = 64 * MEM_LD;

// the three products of every accumulator, kept apart (back to back each would wait for the one before)
__device__ inline void mem_mma3(float (&acc)[8][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[4][4], const uint32_t (&bl)[4][4]) {
    typedef Mma16<__nv_bfloat16> X;
#pragma unroll
    for (int n = 0; n < 4; ++n) { X::mma(acc[2 * n], ah, bh[n][0], bh[n][1]); X::mma(acc[2 * n + 1], ah, bh[n][2], bh[n][3]); }
#pragma unroll
    for (int n = 0; n < 4; ++n) { X::mma(acc[2 * n], ah, bl[n][0], bl[n][1]); X::mma(acc[2 * n + 1], ah, bl[n][2], bl[n][3]); }
#pragma unroll
    for (int n = 0; n < 4; ++n) { X::mma(acc[2 * n], al, bh[n][0], bh[n][1]); X::mma(acc[2 * n + 1], al, bh[n][2], bh[n][3]); }
}

// acc[64 columns] of this warp's 16 rows += A B with three products of the heads and remainders; A fragments from
// `load_a(k, hi, lo)`, B stored [k][64] in (bhi, blo)
template <class LoadA>
__device__ inline void mem_mma_kn(float (&acc)[8][4], uint32_t bhi, uint32_t blo, LoadA load_a) {
    const int lane = threadIdx.x & 31;
    const uint32_t off = (uint32_t)((lane & 7) + 8 * ((lane >> 3) & 1)) * (MEM_LD * 2) + (uint32_t)(8 * (lane >> 4)) * 2u;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        uint32_t ah[4], al[4];
        load_a(k, ah, al);
        uint32_t bh[4][4], bl[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            ldsm_x4_trans(bh[n], bhi + off + (uint32_t)(16 * k) * (MEM_LD * 2) + (uint32_t)n * 32u);
            ldsm_x4_trans(bl[n], blo + off + (uint32_t)(16 * k) * (MEM_LD * 2) + (uint32_t)n * 32u);
        }
        mem_mma3(acc, ah, al, bh, bl);
    }
}

// contributions: grid = (nchunk, H, value blocks x key blocks of 64)
static __global__ void __launch_bounds__(128) mem_chunk_kernel(const __grid_constant__ MemPrompt p, int vblocks) {
    __shared__ __align__(128) __nv_bfloat16 tiles[4 * MEM_TILE_ELEMS];
    __shared__ float F[MEM_CHUNK], I[MEM_CHUNK], W[MEM_CHUNK], tmp;
    const MemDims& d = p.d;
    const int c = blockIdx.x, h = blockIdx.y, vb = blockIdx.z % vblocks, kb = blockIdx.z / vblocks, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int t0 = c * MEM_CHUNK, nt = min(MEM_CHUNK, p.rows - t0);
    mem_chunk_gates(p, h, t0, nt, F, I, &tmp);
    const float Fend = F[MEM_CHUNK - 1];
    const bool linear = d.linear();
    float wmax = linear ? 0.0f : -INFINITY;
    for (int s = 0; s < nt && !linear; ++s) wmax = fmaxf(wmax, Fend - F[s] + I[s]);
    if (tid < MEM_CHUNK) W[tid] = expf(Fend - F[tid] + I[tid] - wmax);
    __syncthreads();
    __nv_bfloat16 *kh = tiles, *kl = tiles + MEM_TILE_ELEMS, *vh = tiles + 2 * MEM_TILE_ELEMS, *vl = tiles + 3 * MEM_TILE_ELEMS;
    const float* row0 = p.proj + (size_t)t0 * p.proj_ld;
    mem_load_tile(kh, kl, row0 + p.pl.rk + h * d.dim + kb * 64, p.proj_ld, nt, d.dim - kb * 64, W, 1.0f);
    mem_load_tile(vh, vl, row0 + p.pl.rv + h * d.vdim + vb * 64, p.proj_ld, nt, d.vdim - vb * 64, nullptr, 1.0f);
    __syncthreads();
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    const uint32_t kha = smem_addr(kh), kla = smem_addr(kl);
    // A = K^T (rows: key dimensions 16 warp ..), K stored [token][dimension]: transposed fragment loads
    const uint32_t a_off = (uint32_t)((lane & 7) + 8 * (lane >> 4)) * (MEM_LD * 2) + (uint32_t)(16 * warp + 8 * ((lane >> 3) & 1)) * 2u;
    mem_mma_kn(acc, smem_addr(vh), smem_addr(vl), [&](int k, uint32_t (&ah)[4], uint32_t (&al)[4]) {
        ldsm_x4_trans(ah, kha + a_off + (uint32_t)(16 * k) * (MEM_LD * 2));
        ldsm_x4_trans(al, kla + a_off + (uint32_t)(16 * k) * (MEM_LD * 2));
    });
    float* U = p.U + ((size_t)c * d.H + h) * d.dim * d.vs;
    const int ra = kb * 64 + 16 * warp + (lane >> 2);
#pragma unroll
    for (int n = 0; n < 8; ++n) {
        const int col = vb * 64 + 8 * n + 2 * (lane & 3);
        if (col < d.vs) {  // vs is even, columns past vdim are zero
            if (ra < d.dim) *reinterpret_cast<float2*>(U + (size_t)ra * d.vs + col) = make_float2(acc[n][0], acc[n][1]);
            if (ra + 8 < d.dim) *reinterpret_cast<float2*>(U + (size_t)(ra + 8) * d.vs + col) = make_float2(acc[n][2], acc[n][3]);
        }
    }
    if (vb == 0) {
        for (int i = tid; i < 64 && kb * 64 + i < d.dim && !linear; i += 128) {
            float s = 0.0f;
            for (int t = 0; t < nt; ++t) s += Elem<__nv_bfloat16>::to_f32(kh[t * MEM_LD + i]) + Elem<__nv_bfloat16>::to_f32(kl[t * MEM_LD + i]);
            p.UN[((size_t)c * d.H + h) * d.dim + kb * 64 + i] = s;
        }
        if (kb == 0 && tid == 0) {
            p.gm[((size_t)c * d.H + h) * 2] = Fend;
            p.gm[((size_t)c * d.H + h) * 2 + 1] = wmax;
            if (c == 0) p.m_live[h] = linear ? 0.0f : p.state[d.m_off() + h * d.nslice];
        }
    }
}

// starting states: grid = (blocks over dim * vs / 4, H) plus one block column (the last) for n and m
static __global__ void __launch_bounds__(256) mem_scan_kernel(const __grid_constant__ MemPrompt p, float* __restrict__ m_start) {
    const MemDims& d = p.d;
    const int h = blockIdx.y, tid = threadIdx.x;
    float m = p.m_live[h];
    if (blockIdx.x + 1 < gridDim.x) {
        const size_t i = (size_t)blockIdx.x * 256 + tid, n4 = (size_t)d.dim * d.vs / 4;
        if (i >= n4) return;
        float4* S = reinterpret_cast<float4*>(p.state + (size_t)h * d.dim * d.vs) + i;
        float4 s = *S;
        const size_t step = (size_t)d.H * n4;
        float4* U = reinterpret_cast<float4*>(p.U) + (size_t)h * n4 + i;
        float4 u = *U;
        for (int c = 0; c < p.nchunk; ++c) {
            const float4 un = c + 1 < p.nchunk ? U[step] : u;  // the next chunk's load does not wait for this one's store
            *U = s;
            const float fe = p.gm[((size_t)c * d.H + h) * 2], w = p.gm[((size_t)c * d.H + h) * 2 + 1];
            const float mn = fmaxf(fe + m, w), a = expf(fe + m - mn), b = expf(w - mn);
            s = make_float4(a * s.x + b * u.x, a * s.y + b * u.y, a * s.z + b * u.z, a * s.w + b * u.w);
            m = mn;
            u = un;
            U += step;
        }
        *S = s;
        return;
    }
    if (d.linear()) return;
    float* nl = p.state + d.n_off() + (size_t)h * d.nslice * d.dim;
    for (int i = tid; i < d.dim; i += 256) {
        float mm = m, s = nl[i];
        for (int c = 0; c < p.nchunk; ++c) {
            float* U = p.UN + ((size_t)c * d.H + h) * d.dim + i;
            const float u = *U;
            *U = s;
            const float fe = p.gm[((size_t)c * d.H + h) * 2], w = p.gm[((size_t)c * d.H + h) * 2 + 1];
            const float mn = fmaxf(fe + mm, w);
            s = expf(fe + mm - mn) * s + expf(w - mn) * u;
            mm = mn;
        }
        for (int k = 0; k < d.nslice; ++k) nl[(size_t)k * d.dim + i] = s;
    }
    if (tid == 0) {
        for (int c = 0; c < p.nchunk; ++c) {
            m_start[(size_t)c * d.H + h] = m;
            m = fmaxf(p.gm[((size_t)c * d.H + h) * 2] + m, p.gm[((size_t)c * d.H + h) * 2 + 1]);
        }
        for (int k = 0; k < d.nslice; ++k) p.state[d.m_off() + h * d.nslice + k] = m;
    }
}

// read-outs: grid = (nchunk, H, value blocks of 64)
constexpr size_t MEM_OUT_SMEM = (size_t)8 * MEM_TILE_ELEMS * 2;
static __global__ void __launch_bounds__(128) mem_out_kernel(const __grid_constant__ MemPrompt p, const float* __restrict__ m_start) {
    extern __shared__ __align__(128) unsigned char mo_raw[];
    __shared__ float F[MEM_CHUNK], I[MEM_CHUNK], Mx[MEM_CHUNK], NQ[MEM_CHUNK], tmp;
    const MemDims& d = p.d;
    const int c = blockIdx.x, h = blockIdx.y, vb = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int t0 = c * MEM_CHUNK, nt = min(MEM_CHUNK, p.rows - t0);
    __nv_bfloat16* t = reinterpret_cast<__nv_bfloat16*>(mo_raw);
    __nv_bfloat16 *qh = t, *ql = t + MEM_TILE_ELEMS, *kh = t + 2 * MEM_TILE_ELEMS, *kl = t + 3 * MEM_TILE_ELEMS;
    __nv_bfloat16 *sh = t + 4 * MEM_TILE_ELEMS, *sl = t + 5 * MEM_TILE_ELEMS, *vh = t + 6 * MEM_TILE_ELEMS, *vl = t + 7 * MEM_TILE_ELEMS;
    mem_chunk_gates(p, h, t0, nt, F, I, &tmp);
    const bool linear = d.linear();
    const float m0 = linear ? 0.0f : m_start[(size_t)c * d.H + h];
    if (linear) {
        if (tid < MEM_CHUNK) Mx[tid] = -F[tid];
    } else if (tid < MEM_CHUNK) {  // M_t by an inclusive maximum scan
        float a = I[tid] - F[tid];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, a, o);
            if ((tid & 31) >= o) a = fmaxf(a, v);
        }
        if (tid == 31) tmp = a;
        Mx[tid] = fmaxf(a, m0);
    }
    __syncthreads();
    if (tid >= 32 && tid < MEM_CHUNK && !linear) Mx[tid] = fmaxf(Mx[tid], tmp);
    const float* row0 = p.proj + (size_t)t0 * p.proj_ld;
    const float* S0 = p.U + ((size_t)c * d.H + h) * d.dim * d.vs;
    const float* N0 = p.UN + ((size_t)c * d.H + h) * d.dim;
    const float qscale = linear ? 1.0f : 1.0f / sqrtf((float)d.dim);
    mem_load_tile(vh, vl, row0 + p.pl.rv + h * d.vdim + vb * 64, p.proj_ld, nt, d.vdim - vb * 64, nullptr, 1.0f);
    float sc[8][4], o[8][4], nq = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const uint32_t a_off = (uint32_t)(16 * warp + (lane & 15)) * (MEM_LD * 2) + (uint32_t)(lane >> 4) * 16u;
    const uint32_t b_off = (uint32_t)((lane & 7) + 8 * (lane >> 4)) * (MEM_LD * 2) + (uint32_t)((lane >> 3) & 1) * 16u;
    for (int kb = 0; kb * 64 < d.dim; ++kb) {
        __syncthreads();  // the previous block's tiles are no longer read
        mem_load_tile(qh, ql, row0 + p.pl.rq + h * d.dim + kb * 64, p.proj_ld, nt, d.dim - kb * 64, nullptr, qscale);
        mem_load_tile(kh, kl, row0 + p.pl.rk + h * d.dim + kb * 64, p.proj_ld, nt, d.dim - kb * 64, nullptr, 1.0f);
        mem_load_tile(sh, sl, S0 + (size_t)kb * 64 * d.vs + vb * 64, d.vs, d.dim - kb * 64, d.vdim - vb * 64, nullptr, 1.0f);
        __syncthreads();
        if (!linear) {   // n_0 . q: two threads per token
            const int tt = tid >> 1, i0 = (tid & 1) * 32;
            for (int i = i0; i < i0 + 32 && kb * 64 + i < d.dim; ++i)
                nq = fmaf(Elem<__nv_bfloat16>::to_f32(qh[tt * MEM_LD + i]) + Elem<__nv_bfloat16>::to_f32(ql[tt * MEM_LD + i]), N0[kb * 64 + i], nq);
        }
        const uint32_t qha = smem_addr(qh), qla = smem_addr(ql), kha = smem_addr(kh), kla = smem_addr(kl);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            uint32_t ah[4], al[4];
            ldsm_x4(ah, qha + a_off + (uint32_t)k * 32u);
            ldsm_x4(al, qla + a_off + (uint32_t)k * 32u);
            uint32_t bh[4][4], bl[4][4];
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                ldsm_x4(bh[n], kha + b_off + (uint32_t)(16 * n) * (MEM_LD * 2) + (uint32_t)k * 32u);
                ldsm_x4(bl[n], kla + b_off + (uint32_t)(16 * n) * (MEM_LD * 2) + (uint32_t)k * 32u);
            }
            mem_mma3(sc, ah, al, bh, bl);
        }
        mem_mma_kn(o, smem_addr(sh), smem_addr(sl), [&](int k, uint32_t (&ah)[4], uint32_t (&al)[4]) {
            ldsm_x4(ah, qha + a_off + (uint32_t)k * 32u);
            ldsm_x4(al, qla + a_off + (uint32_t)k * 32u);
        });
    }
    nq += __shfl_xor_sync(0xffffffffu, nq, 1);
    if ((tid & 1) == 0) NQ[tid >> 1] = nq;
    __syncthreads();
    const int ta = 16 * warp + (lane >> 2), tb = ta + 8, tq = lane & 3;
    const float M_a = Mx[ta], M_b = Mx[tb], e_a = expf(m0 - M_a), e_b = expf(m0 - M_b);
    float n_a = 0.0f, n_b = 0.0f;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int s = 8 * n + 2 * tq + e;
            const float as = I[s] - F[s];
            sc[n][e] = s <= ta ? sc[n][e] * expf(as - M_a) : 0.0f;
            sc[n][2 + e] = s <= tb ? sc[n][2 + e] * expf(as - M_b) : 0.0f;
            n_a += sc[n][e];
            n_b += sc[n][2 + e];
            o[n][e] *= e_a;
            o[n][2 + e] *= e_b;
        }
    }
#pragma unroll
    for (int w = 1; w < 4; w <<= 1) {
        n_a += __shfl_xor_sync(0xffffffffu, n_a, w);
        n_b += __shfl_xor_sync(0xffffffffu, n_b, w);
    }
    mem_mma_kn(o, smem_addr(vh), smem_addr(vl), [&](int k, uint32_t (&ah)[4], uint32_t (&al)[4]) {
        typedef __nv_bfloat16 B;
        const float* s0 = sc[2 * k];
        const float* s1 = sc[2 * k + 1];
        ah[0] = pack2<B>(s0[0], s0[1]); ah[1] = pack2<B>(s0[2], s0[3]); ah[2] = pack2<B>(s1[0], s1[1]); ah[3] = pack2<B>(s1[2], s1[3]);
        al[0] = pack2<B>(s0[0] - round16<B>(s0[0]), s0[1] - round16<B>(s0[1])); al[1] = pack2<B>(s0[2] - round16<B>(s0[2]), s0[3] - round16<B>(s0[3]));
        al[2] = pack2<B>(s1[0] - round16<B>(s1[0]), s1[1] - round16<B>(s1[1])); al[3] = pack2<B>(s1[2] - round16<B>(s1[2]), s1[3] - round16<B>(s1[3]));
    });
    const float d_a = linear ? 1.0f : 1.0f / (fmaxf(fabsf(n_a + e_a * NQ[ta]), expf(-(F[ta] + M_a))) + 1e-6f);
    const float d_b = linear ? 1.0f : 1.0f / (fmaxf(fabsf(n_b + e_b * NQ[tb]), expf(-(F[tb] + M_b))) + 1e-6f);
    const int ld = d.H * d.vdim;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int col = vb * 64 + 8 * n + 2 * tq + e;
            if (col < d.vdim) {
                if (ta < nt) p.out[(size_t)(t0 + ta) * ld + h * d.vdim + col] = o[n][e] * d_a;
                if (tb < nt) p.out[(size_t)(t0 + tb) * ld + h * d.vdim + col] = o[n][2 + e] * d_b;
            }
        }
    }
}

// per token: the read-outs, each head divided by its root mean square (linear attention: all heads by their common one),
// times norm weight and gate, as a GEMM operand
template <typename AT>
__global__ void __launch_bounds__(256) mem_rows_kernel(const float* __restrict__ mem, const float* __restrict__ proj, int proj_ld, int gate_off, MemDims d,
                                                       const float* __restrict__ norm, AT* __restrict__ hi, AT* __restrict__ lo, int ld) {
    __shared__ float red[32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n = d.H * d.vdim;
    const float* row = mem + (size_t)blockIdx.x * n;
    const float* gate = proj + (size_t)blockIdx.x * proj_ld + gate_off;
    auto put = [&](int j, float r) { pf_store(hi, lo, (size_t)blockIdx.x * ld + j, row[j] * r * norm[j] * sigmoid(gate[j])); };
    if (d.linear()) {
        float ss = 0.0f;
        for (int j = threadIdx.x; j < n; j += 256) ss = fmaf(row[j], row[j], ss);
        const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)n + d.eps);
        for (int j = threadIdx.x; j < n; j += 256) put(j, r);
    } else {
        for (int h = warp; h < d.H; h += 8) {
            float ss = 0.0f;
            for (int i = lane; i < d.vdim; i += 32) { const float v = row[h * d.vdim + i]; ss = fmaf(v, v, ss); }
            const float r = 1.0f / sqrtf(warp_sum(ss) / (float)d.vdim + d.eps);
            for (int i = lane; i < d.vdim; i += 32) put(h * d.vdim + i, r);
        }
    }
    for (int j = n + threadIdx.x; j < ld; j += 256) pf_store(hi, lo, (size_t)blockIdx.x * ld + j, 0.0f);
}

// ---------------------------------------------------------------------- residual stream behind a sublayer, one CTA per token
template <typename AT>
__global__ void __launch_bounds__(256) parallel_mix_rows_kernel(float* __restrict__ x, const float* __restrict__ yl, const float* __restrict__ yr, int y_ld,
                                                                const float* __restrict__ wl, const float* __restrict__ wr, const float* __restrict__ gain,
                                                                float mult, float eps, int n, int D, AT* __restrict__ hi, AT* __restrict__ lo) {
    extern __shared__ float mixed[];  // [D]
    __shared__ float red[32];
    const float *a = yl + (size_t)blockIdx.x * y_ld, *b = yr + (size_t)blockIdx.x * y_ld;
    float sl = 0.0f, sr = 0.0f, ss = 0.0f;
    for (int i = threadIdx.x; i < D; i += 256) { sl = fmaf(a[i], a[i], sl); sr = fmaf(b[i], b[i], sr); }
    const float rl = 0.5f / sqrtf(block_sum(sl, red) * (1.0f / (float)n) + eps), rr = 0.5f / sqrtf(block_sum(sr, red) * (1.0f / (float)n) + eps);
    for (int i = threadIdx.x; i < D; i += 256) {
        const float z = a[i] * rl * wl[i] + b[i] * rr * wr[i];
        mixed[i] = z;
        ss = fmaf(z, z, ss);
    }
    const float r = mult / sqrtf(block_sum(ss, red) * (1.0f / (float)n) + eps);
    for (int i = threadIdx.x; i < D; i += 256) {
        const size_t at = (size_t)blockIdx.x * D + i;
        const float v = x[at] + mixed[i] * r * gain[i];
        x[at] = v;
        pf_store(hi, lo, at, v);
    }
}

// mean and reciprocal deviation of the first n entries of a row in shared memory
__device__ inline void row_moments(const float* row, int n, int kind, float eps, float* red, float& mean, float& r) {
    mean = 0.0f;
    if (kind == VecNorm::LAYER) {
        float s = 0.0f;
        for (int i = threadIdx.x; i < n; i += 256) s += row[i];
        mean = block_sum(s, red) * (1.0f / (float)n);
    }
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += 256) { const float v = row[i] - mean; ss = fmaf(v, v, ss); }
    r = 1.0f / sqrtf(block_sum(ss, red) * (1.0f / (float)n) + eps);
}

// x += mult * post(y) + add, and pre(x) as a GEMM operand (InResidual, mixers.cuh).  y: none, one row per token, or (slots !=
// nullptr) the rows of the token's chosen experts, weighted by their scores in the order they were chosen
struct ResidualRows {
    float* x;
    const float* y;
    int y_ld;
    const int* slots;
    const float* weights;
    int top;
    VecNorm post;
    const float* add;
    VecNorm pre;
    float mult, eps;
    int n, D;            // entries the norms are over; zeros follow up to D
};
template <typename AT>
__global__ void __launch_bounds__(256) residual_rows_kernel(ResidualRows p, AT* __restrict__ hi, AT* __restrict__ lo) {
    extern __shared__ float sum[];  // [D]; a thread touches its own entries only
    __shared__ float red[32];
    float mean = 0.0f, r = 1.0f;
    const bool normed = p.y != nullptr && p.post.kind != VecNorm::NONE;
    if (p.y != nullptr) {
        for (int i = threadIdx.x; i < p.D; i += 256) {
            float v = 0.0f;
            if (p.slots != nullptr) {
                for (int k = 0; k < p.top; ++k) v = fmaf(p.weights[blockIdx.x * p.top + k], p.y[(size_t)p.slots[blockIdx.x * p.top + k] * p.y_ld + i], v);
            } else {
                v = p.y[(size_t)blockIdx.x * p.y_ld + i];
            }
            sum[i] = v;
        }
        if (normed) row_moments(sum, p.n, p.post.kind, p.eps, red, mean, r);
    }
    r *= p.mult;
    for (int i = threadIdx.x; i < p.D; i += 256) {
        const size_t at = (size_t)blockIdx.x * p.D + i;
        float v = p.x[at];
        if (normed) v += (sum[i] - mean) * r * p.post.w[i] + (p.post.b != nullptr ? p.mult * p.post.b[i] : 0.0f);
        else if (p.y != nullptr) v += sum[i] * r;
        if (p.add != nullptr) v += p.add[i];
        p.x[at] = v;
        sum[i] = v;
    }
    const bool ahead = p.pre.kind != VecNorm::NONE;
    if (ahead) row_moments(sum, p.n, p.pre.kind, p.eps, red, mean, r);
    for (int i = threadIdx.x; i < p.D; i += 256) {
        float v = sum[i];
        if (ahead) v = (v - mean) * r * p.pre.w[i] + (p.pre.b != nullptr ? p.pre.b[i] : 0.0f);
        pf_store(hi, lo, (size_t)blockIdx.x * p.D + i, v);
    }
}

// ---------------------------------------------------------------------- mixture of experts: routing of all tokens
// four tokens per CTA, one warp each
static __global__ void __launch_bounds__(128) route_rows_kernel(const float* __restrict__ logits, int ld, int rows, RouteRule rule, int* __restrict__ sel_ids,
                                                                float* __restrict__ sel_w) {
    extern __shared__ float rr_sm[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x * 4 + warp;
    if (t >= rows) return;
    float* pr = rr_sm + (size_t)warp * (rule.experts + rule.groups);
    for (int k = lane; k < rule.experts; k += 32) pr[k] = logits[(size_t)t * ld + k];
    __syncwarp();
    route_pick(pr, pr + rule.experts, rule, lane, [&](int k, int e, float w) {
        if (lane == 0) {
            sel_ids[(size_t)t * rule.top + k] = e;
            sel_w[(size_t)t * rule.top + k] = w;
        }
    });
}

// One CTA: rows of the permuted activations.  Expert e owns a run of rows that starts on a multiple of 128 (the GEMM's row
// tile); slots[token * top + k] is where that token's copy for its k-th expert goes, tile_group[tile] the tile's expert.
static __global__ void __launch_bounds__(1024) plan_rows_kernel(const int* __restrict__ sel_ids, int n, int experts, int max_tiles, int* __restrict__ slots,
                                                                int* __restrict__ tile_group) {
    extern __shared__ int plan[];  // [experts] counts, then next free row
    for (int e = threadIdx.x; e < experts; e += 1024) plan[e] = 0;
    for (int i = threadIdx.x; i < max_tiles; i += 1024) tile_group[i] = -1;
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += 1024) atomicAdd(&plan[sel_ids[i]], 1);
    __syncthreads();
    if (threadIdx.x == 0) {
        int tile = 0;
        for (int e = 0; e < experts; ++e) {
            const int tiles = (plan[e] + PF_BM - 1) / PF_BM;
            plan[e] = tile * PF_BM;
            for (int k = 0; k < tiles; ++k) tile_group[tile + k] = e;
            tile += tiles;
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += 1024) slots[i] = atomicAdd(&plan[sel_ids[i]], 1);
}

// copies of the tokens' rows (both parts of the operand) to their slots; grid = rows * top
template <typename AT>
__global__ void __launch_bounds__(128) gather_rows_kernel(const AT* __restrict__ hi, const AT* __restrict__ lo, const int* __restrict__ slots, int top, int D,
                                                          AT* __restrict__ out_hi, AT* __restrict__ out_lo) {
    const size_t src = (size_t)(blockIdx.x / top) * D, dst = (size_t)slots[blockIdx.x] * D;
    constexpr int E = 16 / sizeof(AT);
    for (int c = threadIdx.x; c < D / E; c += 128) {
        *reinterpret_cast<uint4*>(out_hi + dst + c * E) = *reinterpret_cast<const uint4*>(hi + src + c * E);
        if (lo != nullptr) *reinterpret_cast<uint4*>(out_lo + dst + c * E) = *reinterpret_cast<const uint4*>(lo + src + c * E);
    }
}

}  // namespace cd
