// Token mixers and vector pre-steps of the configured decoder (hybrid.h), one token per step.  Each mechanism takes its
// sizes and constants as parameters:
//   softmax attention            a window or the whole context; whole-projection RMS norm of q and k or rotated positions, a
//                                temperature on q that grows with the position, a linear distance bias per head, a sink in
//                                the denominator, a gate per head or per element, key and value widths of their own, paged
//                                cache; one map, or two over the same values with the second one subtracted
//   matrix memory (mLSTM)        S <- f S + i k v^T per head with exponential input gate, sigmoid forget gate and a running
//                                maximum; fp32 state in HBM, updated in place
//   linear attention             the same state with a constant decay per head and neither gates nor normaliser
//   GEMV inputs                  residual + norm of a sublayer's output (+ a vector), followed by the norm ahead of the next
//                                one; the average of two normed outputs; the memory's per-head norm and gate; one norm over
//                                all heads and a gate - folded into the GEMV that consumes the vector
//   GEMV output                  a token's part of a second embedding times an activated gate
// The mixers of a layer run in one launch (mixer_step_kernel); latent attention is in moe.cuh (mla_*).  The routing rule
// shared by the decode router and the batched one is route_pick (moe.cuh).
#pragma once
#include "common.cuh"
#include "kernels.cuh"
#include "moe.cuh"

namespace cd {

// Offsets of the projections in one row of proj [rows]: left (attention) q | k | v | gate, right (memory)
// q | k | v | gate | input gate | forget gate; latent attention has q | latent | key part from lq on.
struct ProjLayout {
    int lq, lk, lv, lg, rq, rk, rv, rg, ri, rf, rows;
};

struct AttnDims {
    int H, G, dim, vdim;
    int kp, vp;          // key (per map) / value row widths in the cache: dim and vdim padded to 16 with zeros
    int maps;            // attention maps per head: a head's query and key are [map][dim]
    int window;          // positions seen, itself included; 0: all
    int page_tokens;
    float scale, eps, temp_coef;
    int temp_every;
    int gate;            // AttnCfg::Gate: 0 none, 1 per head, 2 per element
    float lambda, out_scale;  // two maps: weight of the second, factor behind the head's norm
    Rotation rot;        // rot.dims entries of every map's query and key
    __host__ __device__ int kr() const { return maps * kp; }
    // a page: K [G][page_tokens][maps * kp], then V [G][page_tokens][vp]
    __host__ __device__ size_t page_elems() const { return (size_t)G * page_tokens * (kr() + vp); }
    __host__ __device__ size_t k_at(int page, int g, int off) const { return (size_t)page * page_elems() + ((size_t)g * page_tokens + off) * kr(); }
    __host__ __device__ size_t v_at(int page, int g, int off) const {
        return (size_t)page * page_elems() + (size_t)G * page_tokens * kr() + ((size_t)g * page_tokens + off) * vp;
    }
    __device__ float temperature(int pos) const {
        return temp_coef == 0.0f ? 1.0f : 1.0f + temp_coef * logf((float)((pos + 1) / temp_every) + 1.0f);
    }
};

// State of one layer: S [H][dim][vs], n [H][nslice][dim], m [H][nslice] (the last two of a matrix memory only).  A slice of MEM_SLICE value columns of a head is
// one CTA's work; n and m are kept once per slice (each CTA updates its own copy, so no CTA waits for another).
constexpr int MEM_SLICE = 32;
struct MemDims {
    int H, dim, vdim;
    int vs;              // row stride of S: vdim padded to 4
    int nslice;          // ceil(vdim / MEM_SLICE)
    float cap, eps;
    const float *decay, *log_decay;  // linear attention: constant decay per head, and its logarithm (finite); nullptr: matrix memory
    __host__ __device__ bool linear() const { return decay != nullptr; }
    __host__ __device__ size_t s_floats() const { return (size_t)H * dim * vs; }
    __host__ __device__ size_t n_off() const { return s_floats(); }
    __host__ __device__ size_t m_off() const { return s_floats() + (size_t)H * nslice * dim; }
    __host__ __device__ size_t floats() const { return ((linear() ? s_floats() : m_off() + (size_t)H * nslice) + 63) / 64 * 64; }
};

__device__ inline float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ inline float log_sigmoid(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ inline float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ inline float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ inline float gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z))); }  // sqrt(2 / pi)

// a norm of a vector: divided by its root mean square, or with its mean taken off first; times w, plus b where there is one
struct VecNorm {
    enum Kind { NONE = 0, RMS, LAYER };
    int kind;
    const float *w, *b;
};

// ---------------------------------------------------------------------- inputs of the streamed GEMV (kernels.cuh, GemvIn)
// x' = x + mult * post(y) + add, published; the GEMV's input is pre(x').  y (a sublayer's output) and add may be absent.
// n: entries the norms are over; the vectors are padded with zeros behind them, weights and biases too.
struct InResidual {
    static constexpr bool CUSTOM = true;
    const float *x, *y, *add;
    float* x_out;
    VecNorm post, pre;
    float mult, eps;
    int n;
    // mean and reciprocal deviation of the vector spread over the consumers' registers
    template <int NITER, int EPC>
    __device__ void moments(const float (&v)[NITER][EPC], int kind, int tid, int nchunks, float* red, int group, float& mean, float& r) const {
        const float inv_n = 1.0f / (float)n;
        mean = 0.0f;
        if (kind == VecNorm::LAYER) {
            float s = 0.0f;
#pragma unroll
            for (int i = 0; i < NITER; ++i)
#pragma unroll
                for (int e = 0; e < EPC; ++e) s += v[i][e];  // zero past the end
            mean = consumer_sum(s, red, group) * inv_n;
        }
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            if (tid + i * GEMV_CONSUMERS < nchunks) {
#pragma unroll
                for (int e = 0; e < EPC; ++e) {
                    const float d = (tid + i * GEMV_CONSUMERS) * EPC + e < n ? v[i][e] - mean : 0.0f;
                    ss = fmaf(d, d, ss);
                }
            }
        }
        r = 1.0f / sqrtf(consumer_sum(ss, red, group) * inv_n + eps);
    }
    __device__ static float4 vec4(const float* p, size_t at) { return p != nullptr ? *reinterpret_cast<const float4*>(p + at) : make_float4(0.f, 0.f, 0.f, 0.f); }
    template <int NITER, int EPC>
    __device__ void load(float (&xr)[NITER][EPC], int tid, int nchunks, float* red, int group, bool, bool writer) const {
        constexpr bool EARLY = NITER * EPC <= 32;  // the residual stream is requested together with y where registers allow
        float xe[EARLY ? NITER : 1][EARLY ? EPC : 1];
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < nchunks && y != nullptr) v = __ldcg(reinterpret_cast<const float4*>(y + (size_t)c * EPC + e));
                xr[i][e] = v.x; xr[i][e + 1] = v.y; xr[i][e + 2] = v.z; xr[i][e + 3] = v.w;
                if constexpr (EARLY) {
                    float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (c < nchunks) b = __ldcg(reinterpret_cast<const float4*>(x + (size_t)c * EPC + e));
                    xe[i][e] = b.x; xe[i][e + 1] = b.y; xe[i][e + 2] = b.z; xe[i][e + 3] = b.w;
                }
            }
        }
        float mean = 0.0f, r = 1.0f;
        if (y != nullptr && post.kind != VecNorm::NONE) moments(xr, post.kind, tid, nchunks, red, group, mean, r);
        const bool normed = y != nullptr && post.kind != VecNorm::NONE;
        r *= mult;
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
            if (c >= nchunks) continue;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                const size_t at = (size_t)c * EPC + e;
                float4 b;
                if constexpr (EARLY) b = make_float4(xe[i][e], xe[i][e + 1], xe[i][e + 2], xe[i][e + 3]);
                else b = __ldcg(reinterpret_cast<const float4*>(x + at));
                const float4 w = normed ? vec4(post.w, at) : make_float4(1.f, 1.f, 1.f, 1.f), o = normed ? vec4(post.b, at) : make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 a = vec4(add, at);
                xr[i][e] = b.x + ((xr[i][e] - mean) * r * w.x + mult * o.x) + a.x;
                xr[i][e + 1] = b.y + ((xr[i][e + 1] - mean) * r * w.y + mult * o.y) + a.y;
                xr[i][e + 2] = b.z + ((xr[i][e + 2] - mean) * r * w.z + mult * o.z) + a.z;
                xr[i][e + 3] = b.w + ((xr[i][e + 3] - mean) * r * w.w + mult * o.w) + a.w;
                if (writer) *reinterpret_cast<float4*>(x_out + at) = make_float4(xr[i][e], xr[i][e + 1], xr[i][e + 2], xr[i][e + 3]);
            }
        }
        if (pre.kind == VecNorm::NONE) return;
        moments(xr, pre.kind, tid, nchunks, red, group, mean, r);
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
            if (c >= nchunks) continue;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                const size_t at = (size_t)c * EPC + e;
                const float4 w = vec4(pre.w, at), o = vec4(pre.b, at);
                xr[i][e] = (xr[i][e] - mean) * r * w.x + o.x;
                xr[i][e + 1] = (xr[i][e + 1] - mean) * r * w.y + o.y;
                xr[i][e + 2] = (xr[i][e + 2] - mean) * r * w.z + o.z;
                xr[i][e + 3] = (xr[i][e + 3] - mean) * r * w.w + o.w;
            }
        }
    }
};

// x' = x + mult * gain * z / rms(z),  z = (wl * yl / rms(yl) + wr * yr / rms(yr)) / 2: the same behind two parallel mixers
struct InParallelMix {
    static constexpr bool CUSTOM = true;
    const float *x, *yl, *yr, *wl, *wr, *gain;
    float* x_out;
    float mult, eps;
    int n;
    template <int NITER, int EPC>
    __device__ void load(float (&xr)[NITER][EPC], int tid, int nchunks, float* red, int group, bool, bool writer) const {
        float sl = 0.0f, sr = 0.0f;
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                if (c < nchunks) {
                    const float4 a = __ldcg(reinterpret_cast<const float4*>(yl + (size_t)c * EPC + e)), b = __ldcg(reinterpret_cast<const float4*>(yr + (size_t)c * EPC + e));
                    sl += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
                    sr += b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
                }
            }
        }
        const float rl = 0.5f / sqrtf(consumer_sum(sl, red, group) * (1.0f / (float)n) + eps);
        const float rr = 0.5f / sqrtf(consumer_sum(sr, red, group) * (1.0f / (float)n) + eps);
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < nchunks) {
                    const size_t at = (size_t)c * EPC + e;
                    const float4 a = __ldcg(reinterpret_cast<const float4*>(yl + at)), b = __ldcg(reinterpret_cast<const float4*>(yr + at));
                    const float4 p = *reinterpret_cast<const float4*>(wl + at), q = *reinterpret_cast<const float4*>(wr + at);
                    z = make_float4(a.x * rl * p.x + b.x * rr * q.x, a.y * rl * p.y + b.y * rr * q.y, a.z * rl * p.z + b.z * rr * q.z, a.w * rl * p.w + b.w * rr * q.w);
                }
                xr[i][e] = z.x; xr[i][e + 1] = z.y; xr[i][e + 2] = z.z; xr[i][e + 3] = z.w;
                ss += z.x * z.x + z.y * z.y + z.z * z.z + z.w * z.w;
            }
        }
        const float r = mult / sqrtf(consumer_sum(ss, red, group) * (1.0f / (float)n) + eps);
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
            if (c >= nchunks) continue;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                const size_t at = (size_t)c * EPC + e;
                const float4 b = __ldcg(reinterpret_cast<const float4*>(x + at)), g = *reinterpret_cast<const float4*>(gain + at);
                xr[i][e] = b.x + xr[i][e] * r * g.x; xr[i][e + 1] = b.y + xr[i][e + 1] * r * g.y;
                xr[i][e + 2] = b.z + xr[i][e + 2] * r * g.z; xr[i][e + 3] = b.w + xr[i][e + 3] * r * g.w;
                if (writer) *reinterpret_cast<float4*>(x_out + at) = make_float4(xr[i][e], xr[i][e + 1], xr[i][e + 2], xr[i][e + 3]);
            }
        }
    }
};

// Input of the paired output projections: the first matrix takes the gated attention output as it is; the second takes
// the memory's raw read-out, each head divided by its root mean square (the sums of squares arrive per slice), times
// the norm weight, times the sigmoid of the gate projection.
struct InMixerOutputs {
    static constexpr bool CUSTOM = true;
    const float *attn, *mem, *ssq, *norm, *gate;
    int n, vdim, nslice;
    float eps;
    template <int NITER, int EPC>
    __device__ void load(float (&xr)[NITER][EPC], int tid, int nchunks, float*, int, bool second, bool) const {
        int hcur = -1;
        float rstd = 0.0f;
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < nchunks) v = __ldcg(reinterpret_cast<const float4*>((second ? mem : attn) + (size_t)c * EPC + e));
                xr[i][e] = v.x; xr[i][e + 1] = v.y; xr[i][e + 2] = v.z; xr[i][e + 3] = v.w;
            }
            if (second && c < nchunks) {
#pragma unroll
                for (int e = 0; e < EPC; ++e) {
                    const int j = c * EPC + e;
                    if (j < n) {
                        const int h = j / vdim;
                        if (h != hcur) {
                            float s = 0.0f;
                            for (int k = 0; k < nslice; ++k) s += __ldcg(ssq + h * nslice + k);
                            rstd = 1.0f / sqrtf(s / (float)vdim + eps);
                            hcur = h;
                        }
                        xr[i][e] = xr[i][e] * rstd * norm[j] * sigmoid(__ldcg(gate + j));
                    }
                }
            }
        }
    }
};

// All heads' read-outs divided by their common root mean square, times the norm weight and the sigmoid of the gate projection.
struct InGatedNorm {
    static constexpr bool CUSTOM = true;
    const float *mem, *norm, *gate;
    int n;
    float eps;
    template <int NITER, int EPC>
    __device__ void load(float (&xr)[NITER][EPC], int tid, int nchunks, float* red, int group, bool, bool) const {
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
#pragma unroll
            for (int e = 0; e < EPC; e += 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < nchunks) v = __ldcg(reinterpret_cast<const float4*>(mem + (size_t)c * EPC + e));
                xr[i][e] = v.x; xr[i][e + 1] = v.y; xr[i][e + 2] = v.z; xr[i][e + 3] = v.w;
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (c * EPC + e + k < n) ss = fmaf(xr[i][e + k], xr[i][e + k], ss);  // another layer's values may lie behind the last head
            }
        }
        const float r = 1.0f / sqrtf(consumer_sum(ss, red, group) / (float)n + eps);
#pragma unroll
        for (int i = 0; i < NITER; ++i) {
            const int c = tid + i * GEMV_CONSUMERS;
            if (c >= nchunks) continue;
#pragma unroll
            for (int e = 0; e < EPC; ++e) {
                const int j = c * EPC + e;
                xr[i][e] = j < n ? xr[i][e] * r * norm[j] * sigmoid(__ldcg(gate + j)) : 0.0f;
            }
        }
    }
};

// One column of a token's part of a second embedding, times the activated gate.
template <typename WT> struct EpiTokenGate {
    float* out;
    const WT* table;   // this layer's first column
    int ld, vocab;
    const DevState* st;
    __device__ void operator()(int unit, const float (&y)[1]) const {
        const uint32_t tok = __ldcg(&st->token);
        out[unit] = gelu_tanh(y[0]) * Elem<WT>::to_f32(table[(size_t)(tok < (uint32_t)vocab ? tok : 0u) * ld + unit]);
    }
};

// The residual stream after the last layer as a vector in memory (one CTA); widths up to 16384.
template <class In>
__global__ void __launch_bounds__(GEMV_CONSUMERS) vector_input_kernel(In in, int n) {
    __shared__ float red[32];
    pdl_wait();
    pdl_launch_dependents();
    if (n <= 4 * 4 * GEMV_CONSUMERS) {
        float xr[4][4];
        in.load(xr, threadIdx.x, n / 4, red, 0, false, true);
    } else {
        float xr[16][4];
        in.load(xr, threadIdx.x, n / 4, red, 0, false, true);
    }
}

// ---------------------------------------------------------------------- one token through both mixers of a layer
struct MixerStep {
    AttnDims a;
    MemDims d;
    ProjLayout pl;
    const float* proj;                 // this token's projections
    const float *q_norm, *k_norm, *sink, *slopes;  // absent ones are nullptr
    const float *ib, *fb;
    const int* page_table;
    const DevState* st;
    float *part_acc, *part_ml;         // [H][maps][nsplit][vp], [H][maps][nsplit][2]
    unsigned int* counters;            // [H]
    float* attn;                       // [H * vdim], gated
    float* mem;                        // [Hr * vdim], raw read-out
    float* ssq;                        // [Hr][nslice]
    float* state;                      // this layer's state
    int nsplit;
};
constexpr int MIX_THREADS = 128, MIX_TILE = 32;
__host__ __device__ inline size_t mixer_attn_smem_floats(int kr, int vp, int maps) { return (size_t)2 * kr + vp + (size_t)MIX_THREADS * 8 + (4 + maps) * MIX_TILE + 96; }
__host__ __device__ inline size_t mixer_mem_smem_floats(int dim) { return (size_t)2 * dim + 4 * MEM_SLICE + 64; }

// this thread's share of the sum of squares of n floats another kernel wrote
__device__ inline float sum_of_squares(const float* v, int n) {
    float s = 0.0f;
    if ((n & 3) == 0 && (reinterpret_cast<size_t>(v) & 15) == 0) {
        const float4* v4 = reinterpret_cast<const float4*>(v);
#pragma unroll 8
        for (int i = threadIdx.x; i < n / 4; i += MIX_THREADS) {
            const float4 t = __ldcg(v4 + i);
            s += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w;
        }
    } else {
#pragma unroll 8
        for (int i = threadIdx.x; i < n; i += MIX_THREADS) { const float t = __ldcg(v + i); s = fmaf(t, t, s); }
    }
    return s;
}

// A matrix-memory slice: MEM_SLICE value columns of one head.  128 threads = 16 row groups x 8 column quads.
__device__ inline void mem_step(const MixerStep& p, int idx, float* sm, float* red) {
    const MemDims& d = p.d;
    const int h = idx / d.nslice, sl = idx % d.nslice, tid = threadIdx.x;
    const int rg = tid >> 3, col = sl * MEM_SLICE + (tid & 7) * 4;
    float* S = p.state + (size_t)h * d.dim * d.vs + col;
    float* nvec = p.state + d.n_off() + ((size_t)h * d.nslice + sl) * d.dim;
    float* mrun = p.state + d.m_off() + h * d.nslice + sl;
    const bool live = col < d.vdim;
    // this CTA's part of the state was written a whole token ago: its first rows are requested before the previous
    // kernel of the chain has finished (at most two neighbours of the chain overlap)
    constexpr int PRE = 8;
    float4 s[PRE];
#pragma unroll
    for (int j = 0; j < PRE; ++j) {
        const int r = rg + 16 * j;
        s[j] = live && r < d.dim ? __ldcg(reinterpret_cast<const float4*>(S + (size_t)r * d.vs)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    pdl_launch_dependents();
    float* qs = sm;
    float* ks = sm + d.dim;
    float* acc_s = sm + 2 * d.dim;  // [4 warps][MEM_SLICE]
    const bool linear = d.linear();
    float mt = 0.0f, fa, ia = 1.0f, qscale = 1.0f;
    if (linear) {
        fa = d.decay[h];
    } else {
        const float zi = __ldcg(p.proj + p.pl.ri + h) + p.ib[h], zf = __ldcg(p.proj + p.pl.rf + h) + p.fb[h];
        const float gi = soft_cap(zi, d.cap), gf = log_sigmoid(soft_cap(zf, d.cap)), m0 = __ldcg(mrun);
        mt = fmaxf(gf + m0, gi);
        fa = expf(gf + m0 - mt);
        ia = expf(gi - mt);
        qscale = 1.0f / sqrtf((float)d.dim);
    }
    float nq = 0.0f;
#pragma unroll 2
    for (int i = tid; i < d.dim; i += MIX_THREADS) {
        float q = __ldcg(p.proj + p.pl.rq + h * d.dim + i) * qscale, k = __ldcg(p.proj + p.pl.rk + h * d.dim + i);
        if (linear) { q = silu(q); k = silu(k); }
        qs[i] = q;
        ks[i] = k;
        if (linear) continue;
        const float nn = fa * __ldcg(nvec + i) + ia * k;
        nvec[i] = nn;
        nq = fmaf(nn, q, nq);
    }
    nq = block_sum(nq, red);  // (its barriers publish qs and ks)
    if (tid == 0 && !linear) *mrun = mt;
    float v[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        v[e] = col + e < d.vdim ? ia * __ldcg(p.proj + p.pl.rv + h * d.vdim + col + e) : 0.0f;
        if (linear) v[e] = silu(v[e]);  // silu(0) = 0
    }
    for (int r0 = rg; r0 < d.dim; r0 += 16 * PRE) {
        if (r0 != rg) {
#pragma unroll
            for (int j = 0; j < PRE; ++j) {
                const int r = r0 + 16 * j;
                s[j] = live && r < d.dim ? __ldcg(reinterpret_cast<const float4*>(S + (size_t)r * d.vs)) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
#pragma unroll
        for (int j = 0; j < PRE; ++j) {
            const int r = r0 + 16 * j;
            if (r < d.dim) {
                const float k = ks[r], q = qs[r];
                const float4 t = make_float4(fmaf(fa, s[j].x, k * v[0]), fmaf(fa, s[j].y, k * v[1]), fmaf(fa, s[j].z, k * v[2]), fmaf(fa, s[j].w, k * v[3]));
                if (live) *reinterpret_cast<float4*>(S + (size_t)r * d.vs) = t;
                acc[0] = fmaf(q, t.x, acc[0]); acc[1] = fmaf(q, t.y, acc[1]); acc[2] = fmaf(q, t.z, acc[2]); acc[3] = fmaf(q, t.w, acc[3]);
            }
        }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 8);
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 16);
    }
    if ((tid & 31) < 8) {
#pragma unroll
        for (int e = 0; e < 4; ++e) acc_s[(tid >> 5) * MEM_SLICE + (tid & 7) * 4 + e] = acc[e];
    }
    __syncthreads();
    if (tid < MEM_SLICE) {
        const int c = sl * MEM_SLICE + tid;
        const float num = acc_s[tid] + acc_s[MEM_SLICE + tid] + acc_s[2 * MEM_SLICE + tid] + acc_s[3 * MEM_SLICE + tid];
        const float o = linear ? num : num / (fmaxf(fabsf(nq), expf(-mt)) + 1e-6f);
        if (c < d.vdim) p.mem[h * d.vdim + c] = o;
        const float ss = warp_sum(c < d.vdim ? o * o : 0.0f);
        if (tid == 0) p.ssq[h * d.nslice + sl] = ss;
    }
}

// One head's slice of the visible positions: scores of MIX_TILE positions at a time, running softmax, weighted values (both
// maps of a differential head over the same values); slices are merged by the CTA of the head that arrives last (a
// counter, nobody waits), which adds the sink, subtracts the second map, norms and applies the gate.
template <typename KT, int MAPS>
__device__ inline void attn_step(const MixerStep& p, KT* __restrict__ pool, int idx, float* sm, float* red, int& s_last) {
    constexpr int EPC = Elem<KT>::EPC;
    constexpr float NEG = -3.402823466e+38f;
    const AttnDims& a = p.a;
    const int h = idx / p.nsplit, sl = idx % p.nsplit, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int gqa = a.H / a.G, g = h / gqa, kr = MAPS * a.kp;
    size_t* k_off = reinterpret_cast<size_t*>(sm);  // [MIX_TILE] where the key and value rows of the tile's positions are
    size_t* v_off = k_off + MIX_TILE;
    float* qs = sm + 4 * MIX_TILE;        // [MAPS][kp] query as it meets the keys: norm, rotation, temperature and scale folded in
    float* kc = qs + kr;                  // [MAPS][kp] this position's key as the cache holds it
    float* vc = kc + kr;                  // [vp]
    float* accs = vc + a.vp;              // [128 threads][8]
    float* ps = accs + MIX_THREADS * 8;   // [MAPS][MIX_TILE]
    pdl_wait();
    pdl_launch_dependents();
    const int pos = __ldcg(&p.st->pos);
    const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0, len = pos + 1 - lo;
    int per = (len + p.nsplit - 1) / p.nsplit;
    per = (per + MIX_TILE - 1) / MIX_TILE * MIX_TILE;
    const int t0 = lo + sl * per, t1 = min(pos + 1, t0 + per);
    float m[MAPS], l[MAPS], acc[MAPS][8];
#pragma unroll
    for (int q = 0; q < MAPS; ++q) {
        m[q] = NEG;
        l[q] = 0.0f;
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[q][e] = 0.0f;
    }
    const int nvc = a.vp / EPC;           // value chunks of a row
    int lv = 1;
    while (lv < nvc) lv <<= 1;            // lanes that share a row of values
    const int vch = tid % lv, vgrp = tid / lv, vgroups = MIX_THREADS / lv;
    if (t0 < t1) {
        const bool newest = t1 == pos + 1;  // this slice holds the current position
        auto locate = [&](int tb) {
            if (tid < MIX_TILE) {
                const int t = min(tb + tid, pos), page = p.page_table[t / a.page_tokens], off = t % a.page_tokens;
                k_off[tid] = a.k_at(page, g, off);
                v_off[tid] = a.v_at(page, g, off);
            }
        };
        locate(t0);
        float rq = a.temperature(pos) * a.scale, rk = 1.0f;
        if (p.q_norm != nullptr) {
            const float sq = sum_of_squares(p.proj + p.pl.lq, a.H * MAPS * a.dim), sk = newest ? sum_of_squares(p.proj + p.pl.lk, a.G * MAPS * a.dim) : 0.0f;
            rq /= sqrtf(block_sum(sq, red) / (float)(a.H * MAPS * a.dim) + a.eps);
            if (newest) rk = 1.0f / sqrtf(block_sum(sk, red) / (float)(a.G * MAPS * a.dim) + a.eps);
        }
        // entry i of head `head`'s [map][kp] vector out of the projections at `src`
        auto entry = [&](const float* src, const float* norm, int head, int i, float r) {
            const int q = i / a.kp, d = i % a.kp, at = (head * MAPS + q) * a.dim;
            if (d >= a.dim) return 0.0f;
            return a.rot.entry(d, [&](int k) { return a.rot.at(pos, k); }, [&](int j) { return __ldcg(src + at + j) * r * (norm != nullptr ? norm[at + j] : 1.0f); });
        };
        for (int i = tid; i < kr; i += MIX_THREADS) qs[i] = entry(p.proj + p.pl.lq, p.q_norm, h, i, rq);
        if (newest) {
            const int page = p.page_table[pos / a.page_tokens], off = pos % a.page_tokens;
            const bool writer = h % gqa == 0;
            for (int i = tid; i < kr; i += MIX_THREADS) {
                const KT v = Elem<KT>::from_f32(entry(p.proj + p.pl.lk, p.k_norm, g, i, rk));
                kc[i] = Elem<KT>::to_f32(v);
                if (writer) pool[a.k_at(page, g, off) + i] = v;
            }
            for (int i = tid; i < a.vp; i += MIX_THREADS) {
                const KT v = Elem<KT>::from_f32(i < a.vdim ? __ldcg(p.proj + p.pl.lv + g * a.vdim + i) : 0.0f);
                vc[i] = Elem<KT>::to_f32(v);
                if (writer) pool[a.v_at(page, g, off) + i] = v;
            }
        }
        __syncthreads();
        const int nkc = a.kp / EPC;
        int lk = 1;
        while (lk < nkc && lk < 32) lk <<= 1;  // lanes that share a key row
        const int kch = lane % lk, side = 32 / lk;
        const float slope = p.slopes != nullptr ? p.slopes[h] : 0.0f;
        for (int tb = t0; tb < t1; tb += MIX_TILE) {
            const int nt = min(MIX_TILE, t1 - tb);
            // the tile's value rows are requested before its scores are worked out
            constexpr int PRE = 4;
            uint4 vw[PRE];
#pragma unroll
            for (int u = 0; u < PRE; ++u) {
                const int j = vgrp + u * vgroups;
                vw[u] = make_uint4(0, 0, 0, 0);
                if (vch < nvc && j < nt && tb + j != pos) vw[u] = ldg_stream_coherent(pool + v_off[j] + (size_t)vch * EPC);
            }
            // scores: warp w takes positions tb + 8 w .. + 7
            for (int j0 = 0; j0 < 8; j0 += 4 * side) {
                float d[4][MAPS];
#pragma unroll
                for (int u = 0; u < 4; ++u)
#pragma unroll
                    for (int q = 0; q < MAPS; ++q) d[u][q] = 0.0f;
                for (int c = kch; c < nkc; c += lk) {
                    uint4 w[4][MAPS];
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        const int j = j0 + u * side + lane / lk, t = tb + 8 * warp + j;
                        const bool cached = j < 8 && t < t1 && t != pos;
                        const KT* row = pool + (cached ? k_off[8 * warp + j] : 0) + (size_t)c * EPC;
#pragma unroll
                        for (int q = 0; q < MAPS; ++q) w[u][q] = cached ? ldg_stream_coherent(row + (size_t)q * a.kp) : make_uint4(0, 0, 0, 0);
                    }
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        const int j = j0 + u * side + lane / lk, t = tb + 8 * warp + j;
#pragma unroll
                        for (int q = 0; q < MAPS; ++q) {
                            float f[EPC];
                            Elem<KT>::unpack(w[u][q], f);
                            if (t == pos) {
#pragma unroll
                                for (int e = 0; e < EPC; ++e) f[e] = kc[q * a.kp + c * EPC + e];
                            }
#pragma unroll
                            for (int e = 0; e < EPC; ++e) d[u][q] = fmaf(qs[q * a.kp + c * EPC + e], f[e], d[u][q]);
                        }
                    }
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) {
#pragma unroll
                    for (int q = 0; q < MAPS; ++q) {
                        for (int o = lk >> 1; o > 0; o >>= 1) d[u][q] += __shfl_xor_sync(0xffffffffu, d[u][q], o);
                        const int j = j0 + u * side + lane / lk;
                        if (kch == 0 && j < 8) ps[q * MIX_TILE + 8 * warp + j] = d[u][q];
                    }
                }
            }
            __syncthreads();
            // every warp takes the tile's 32 scores, one per lane
            const int t = tb + lane;
            float pr[MAPS], corr[MAPS];
#pragma unroll
            for (int q = 0; q < MAPS; ++q) {
                const float sc = t < t1 ? ps[q * MIX_TILE + lane] - slope * (float)(pos - t) : NEG;
                const float mn = fmaxf(m[q], warp_max(sc));
                pr[q] = t < t1 ? expf(sc - mn) : 0.0f;
                corr[q] = expf(m[q] - mn);
                l[q] = l[q] * corr[q] + warp_sum(pr[q]);
                m[q] = mn;
            }
            __syncthreads();
            if (warp == 0) {
#pragma unroll
                for (int q = 0; q < MAPS; ++q) ps[q * MIX_TILE + lane] = pr[q];
            }
            __syncthreads();
#pragma unroll
            for (int q = 0; q < MAPS; ++q)
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[q][e] *= corr[q];
            if (vch < nvc) {
                auto add = [&](int j, const uint4& raw) {
                    float f[EPC];
                    Elem<KT>::unpack(raw, f);
                    if (tb + j == pos) {
#pragma unroll
                        for (int e = 0; e < EPC; ++e) f[e] = vc[vch * EPC + e];
                    }
#pragma unroll
                    for (int q = 0; q < MAPS; ++q) {
                        const float w = ps[q * MIX_TILE + j];
#pragma unroll
                        for (int e = 0; e < EPC; ++e) acc[q][e] = fmaf(w, f[e], acc[q][e]);
                    }
                };
#pragma unroll
                for (int u = 0; u < PRE; ++u)
                    if (vgrp + u * vgroups < nt) add(vgrp + u * vgroups, vw[u]);
#pragma unroll 4
                for (int j = vgrp + PRE * vgroups; j < nt; j += vgroups)
                    add(j, tb + j == pos ? make_uint4(0, 0, 0, 0) : ldg_stream_coherent(pool + v_off[j] + (size_t)vch * EPC));
            }
            __syncthreads();  // the tile's places and probabilities are no longer read
            if (tb + MIX_TILE < t1) {
                locate(tb + MIX_TILE);
                __syncthreads();
            }
        }
#pragma unroll
        for (int q = 0; q < MAPS; ++q) {
            if (q > 0) __syncthreads();
#pragma unroll
            for (int e = 0; e < 8; ++e) accs[tid * 8 + e] = acc[q][e];
            __syncthreads();
            float* pa = p.part_acc + ((size_t)(h * MAPS + q) * p.nsplit + sl) * a.vp;
            for (int i = tid; i < a.vp; i += MIX_THREADS) {
                float s = 0.0f;
                for (int gg = 0; gg < vgroups; ++gg) s += accs[(gg * lv + i / EPC) * 8 + i % EPC];
                pa[i] = s;
            }
        }
    }
    if (tid == 0) {
#pragma unroll
        for (int q = 0; q < MAPS; ++q) {
            p.part_ml[((size_t)(h * MAPS + q) * p.nsplit + sl) * 2] = m[q];
            p.part_ml[((size_t)(h * MAPS + q) * p.nsplit + sl) * 2 + 1] = l[q];
        }
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) s_last = atomicAdd(&p.counters[h], 1u) == (unsigned)p.nsplit - 1u;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    float inv[MAPS];
#pragma unroll
    for (int q = 0; q < MAPS; ++q) {
        const float* pml = p.part_ml + (size_t)(h * MAPS + q) * p.nsplit * 2;
        float ms = NEG, ls = 0.0f;  // nsplit <= 32: one slice per lane, the same in every warp
        if (lane < p.nsplit) {
            const float2 ml = __ldcg(reinterpret_cast<const float2*>(pml + lane * 2));
            ms = ml.x;
            ls = ml.y;
        }
        const float sink = p.sink != nullptr ? p.sink[h] : NEG;
        const float M = fmaxf(warp_max(ls > 0.0f ? ms : NEG), sink);
        const float w = ls > 0.0f ? expf(ms - M) : 0.0f;
        inv[q] = 1.0f / (warp_sum(ls * w) + (p.sink != nullptr ? expf(sink - M) : 0.0f));
        if (warp == 0) ps[q * MIX_TILE + lane] = w;
    }
    if (MAPS > 1) inv[MAPS - 1] *= -a.lambda;
    __syncthreads();
    const int used = (len + per - 1) / per;  // slices that hold positions
    float ss = 0.0f;
    for (int i = tid; i < a.vdim; i += MIX_THREADS) {
        float r = 0.0f;
#pragma unroll
        for (int q = 0; q < MAPS; ++q) {
            const float* pa = p.part_acc + (size_t)(h * MAPS + q) * p.nsplit * a.vp + i;
            float o = 0.0f;
            for (int s0 = 0; s0 < used; s0 += 16) {  // sixteen slices in flight together
                float t[16];
#pragma unroll
                for (int s = 0; s < 16; ++s) t[s] = s0 + s < used ? __ldcg(pa + (size_t)(s0 + s) * a.vp) : 0.0f;
#pragma unroll
                for (int s = 0; s < 16; ++s)
                    if (s0 + s < used) o = fmaf(t[s], ps[q * MIX_TILE + s0 + s], o);
            }
            r = fmaf(o, inv[q], r);
        }
        vc[i] = r;  // each thread reads its own entries again
        ss = fmaf(r, r, ss);
    }
    float f = MAPS > 1 ? a.out_scale / sqrtf(block_sum(ss, red) / (float)a.vdim + a.eps) : 1.0f;
    if (a.gate == 1) f *= sigmoid(__ldcg(p.proj + p.pl.lg + h));
    for (int i = tid; i < a.vdim; i += MIX_THREADS)
        p.attn[h * a.vdim + i] = vc[i] * f * (a.gate == 2 ? sigmoid(__ldcg(p.proj + p.pl.lg + h * a.vdim + i)) : 1.0f);
    if (tid == 0) p.counters[h] = 0u;
}

// grid = Hr * nslice memory CTAs, then H * nsplit attention CTAs (H or Hr is 0 in a layer with one mixer)
template <typename KT, int MAPS>
__global__ void __launch_bounds__(MIX_THREADS) mixer_step_kernel(const __grid_constant__ MixerStep p, KT* __restrict__ pool) {
    extern __shared__ float mix_sm[];
    __shared__ float red[32];
    __shared__ int s_last;
    const int nmem = p.d.H * p.d.nslice;
    if ((int)blockIdx.x < nmem) mem_step(p, blockIdx.x, mix_sm, red);
    else attn_step<KT, MAPS>(p, pool, blockIdx.x - nmem, mix_sm, red, s_last);
}

}  // namespace cd
