// hybrid_linear.cu — kernels around the linear-attention recurrences of the hybrid decoder family (API: hybrid_kernels.hpp): operands of
// gated linear attention (a decay per key channel), retention (a fixed decay per head, rotate-half rotary), HGRN2 (a forget gate with a lower
// bound whose complement is what is written) and the xLSTM matrix memory (log gates, running maximum, normaliser); the norm after the sum that closes a sublayer of a post-norm design; the router that reads a token's
// experts from a table.  The recurrences themselves are hy_recurrence (hybrid_kernels.cu).  Everything here is fp32 arithmetic; TA is the
// element type of projection outputs and of the rows handed to the next matrix product.
#include <algorithm>

#include "hybrid_common.cuh"
#include "hybrid_kernels.hpp"

namespace oa {

namespace {

using namespace hyk;

__device__ __forceinline__ float log_sigmoidf_(float z) { return z >= 0.f ? -log1pf(expf(-z)) : z - log1pf(expf(z)); }

// ---------------------------------------------------------------------------------------------------------------------------------
// norm after the sum
// ---------------------------------------------------------------------------------------------------------------------------------
template <typename TA>
__global__ void __launch_bounds__(256) hy_post_norm_kernel(float* __restrict__ x, float beta, const float* __restrict__ y1, const float* __restrict__ rw1,
                                                           const float* __restrict__ y2, const float* __restrict__ rw2, float branch_scale, const float* __restrict__ w,
                                                           TA* __restrict__ h, int ldh, int W, float eps) {
    HY_PDL();
    __shared__ float red[32];
    const long long t = blockIdx.x;
    float* xr = x + t * W; const float* a = y1 ? y1 + t * W : nullptr; const float* b = y2 ? y2 + t * W : nullptr;
    float r1 = 1.f, r2 = 1.f;
    if (rw1) {                                   // two sublayers side by side: each output RMS-normed over the width
        float s1 = 0.f, s2 = 0.f;
        for (int c = threadIdx.x; c < W; c += blockDim.x) { s1 = fmaf(a[c], a[c], s1); s2 = fmaf(b[c], b[c], s2); }
        r1 = 1.0f / sqrtf(block_sum(s1, red) / (float)W + eps); r2 = 1.0f / sqrtf(block_sum(s2, red) / (float)W + eps);
    }
    auto val = [&](int c) -> float {
        float v = beta * xr[c];
        if (rw1) v += branch_scale * (a[c] * r1 * rw1[c] + b[c] * r2 * rw2[c]);
        else if (a) v += a[c];
        return v;
    };
    float s = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) s += val(c);
    const float mean = block_sum(s, red) / (float)W;
    float q = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) { const float d = val(c) - mean; q = fmaf(d, d, q); }
    const float rstd = 1.0f / sqrtf(block_sum(q, red) / (float)W + eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) {          // a thread rewrites only what it alone has read
        const float o = (val(c) - mean) * rstd * w[c];
        xr[c] = o;
        if (h) stf(h + t * ldh + c, o);
    }
}

// The same with the row in registers (W a multiple of 4 up to 8192, 16-byte aligned rows): every input is read once, 16 bytes per access.
// The sums run per thread over its own float4s and then over the block, as in the form above with another assignment of channels to
// threads; a model takes one of the two forms for all of its steps.
__device__ __forceinline__ void st4a(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4a(__nv_bfloat16* p, const float4& v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
template <typename TA, int NV>      // NV float4 per thread: W <= 1024 NV
__global__ void __launch_bounds__(256) hy_post_norm_reg_kernel(float* __restrict__ x, float beta, const float* __restrict__ y1, const float* __restrict__ rw1,
                                                               const float* __restrict__ y2, const float* __restrict__ rw2, float branch_scale, const float* __restrict__ w,
                                                               TA* __restrict__ h, int ldh, int W, float eps) {
    HY_PDL();
    __shared__ float red[32];
    const long long t = blockIdx.x;
    const int n4 = W / 4;
    float4* xr = reinterpret_cast<float4*>(x + t * W);
    const float4* a = y1 ? reinterpret_cast<const float4*>(y1 + t * W) : nullptr; const float4* b = y2 ? reinterpret_cast<const float4*>(y2 + t * W) : nullptr;
    float4 v[NV];
    if (rw1) {
        float4 u[NV]; float s1 = 0.f, s2 = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = threadIdx.x + k * 256;
            if (i < n4) { v[k] = a[i]; u[k] = b[i]; s1 += (v[k].x * v[k].x + v[k].y * v[k].y) + (v[k].z * v[k].z + v[k].w * v[k].w); s2 += (u[k].x * u[k].x + u[k].y * u[k].y) + (u[k].z * u[k].z + u[k].w * u[k].w); }
        }
        const float r1 = branch_scale / sqrtf(block_sum(s1, red) / (float)W + eps), r2 = branch_scale / sqrtf(block_sum(s2, red) / (float)W + eps);
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = threadIdx.x + k * 256;
            if (i < n4) {
                const float4 g1 = reinterpret_cast<const float4*>(rw1)[i], g2 = reinterpret_cast<const float4*>(rw2)[i], xv = xr[i];
                v[k].x = fmaf(beta, xv.x, v[k].x * r1 * g1.x + u[k].x * r2 * g2.x); v[k].y = fmaf(beta, xv.y, v[k].y * r1 * g1.y + u[k].y * r2 * g2.y);
                v[k].z = fmaf(beta, xv.z, v[k].z * r1 * g1.z + u[k].z * r2 * g2.z); v[k].w = fmaf(beta, xv.w, v[k].w * r1 * g1.w + u[k].w * r2 * g2.w);
            }
        }
    } else {
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = threadIdx.x + k * 256;
            if (i < n4) {
                const float4 xv = xr[i]; const float4 yv = a ? a[i] : make_float4(0.f, 0.f, 0.f, 0.f);
                v[k] = make_float4(fmaf(beta, xv.x, yv.x), fmaf(beta, xv.y, yv.y), fmaf(beta, xv.z, yv.z), fmaf(beta, xv.w, yv.w));
            }
        }
    }
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) if (threadIdx.x + k * 256 < n4) s += (v[k].x + v[k].y) + (v[k].z + v[k].w);
    const float mean = block_sum(s, red) / (float)W;
    float q = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) if (threadIdx.x + k * 256 < n4) { const float c0 = v[k].x - mean, c1 = v[k].y - mean, c2 = v[k].z - mean, c3 = v[k].w - mean; q += (c0 * c0 + c1 * c1) + (c2 * c2 + c3 * c3); }
    const float rstd = 1.0f / sqrtf(block_sum(q, red) / (float)W + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = threadIdx.x + k * 256;
        if (i < n4) {
            const float4 g = reinterpret_cast<const float4*>(w)[i];
            const float4 o = make_float4((v[k].x - mean) * rstd * g.x, (v[k].y - mean) * rstd * g.y, (v[k].z - mean) * rstd * g.z, (v[k].w - mean) * rstd * g.w);
            xr[i] = o;
            if (h) st4a(h + t * ldh + 4 * i, o);
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------------------------
// operands of the recurrences
// ---------------------------------------------------------------------------------------------------------------------------------
template <typename TA>
__global__ void __launch_bounds__(128) hy_lin_prep_kernel(HyLinPrep p, const TA* __restrict__ q, const TA* __restrict__ k, const TA* __restrict__ v, int ld,
                                                          float* __restrict__ qq, float* __restrict__ kk, float* __restrict__ vv, float* __restrict__ dec_channel, float inv_tau,
                                                          const float* __restrict__ decay_head, float* __restrict__ dec_head, const float* __restrict__ rope_cos,
                                                          const float* __restrict__ rope_sin, HyRows r) {
    HY_PDL();
    const long long t = blockIdx.x;
    const int H = p.heads, D = p.dim, VD = p.vdim, half = p.rot_dims / 2, pos = r.positions[t];
    const float sc = rsqrtf((float)D), qs = p.q_scaled ? sc : 1.f, ks = p.k_scaled ? sc : 1.f;
    const TA* qr = q + t * ld; const TA* kr = k + t * ld;
    for (int i = threadIdx.x; i < H * D; i += blockDim.x) {
        const int d = i % D;
        float a = ldf(qr + i), b = ldf(kr + i);
        if (d < p.rot_dims) {                    // channel d pairs with d + half: (u, v) -> (u cos - v sin, v cos + u sin)
            const bool lo = d < half; const int j = lo ? d : d - half;
            const float c = rope_cos[(long long)pos * half + j], s = rope_sin[(long long)pos * half + j];
            const float ao = ldf(qr + (lo ? i + half : i - half)), bo = ldf(kr + (lo ? i + half : i - half));
            a = lo ? a * c - ao * s : a * c + ao * s;
            b = lo ? b * c - bo * s : b * c + bo * s;
        }
        qq[t * H * D + i] = a * qs; kk[t * H * D + i] = b * ks;
        if (dec_channel) dec_channel[t * H * D + i] = expf(log_sigmoidf_(dec_channel[t * H * D + i]) * inv_tau);
    }
    for (int i = threadIdx.x; i < H * VD; i += blockDim.x) vv[t * H * VD + i] = ldf(v + t * ld + i);
    if (dec_head) for (int i = threadIdx.x; i < H; i += blockDim.x) dec_head[t * H + i] = decay_head[i];
}

// The same for bf16 rows whose heads come in aligned groups of 8 channels (dim, vdim, rot_dims / 2 multiples of 8): a thread owns 8 channels,
// every access is 16 bytes wide.  k_gate (matrix memory): k is multiplied by k_gate[t, head].  Per element the arithmetic is that of the
// kernels above and below: the same bits.
__global__ void __launch_bounds__(128) hy_lin_prep_vec8_kernel(HyLinPrep p, const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k, const __nv_bfloat16* __restrict__ v,
                                                               int ld, float* __restrict__ qq, float* __restrict__ kk, float* __restrict__ vv, float* __restrict__ dec_channel,
                                                               float inv_tau, const float* __restrict__ decay_head, float* __restrict__ dec_head, const float* __restrict__ rope_cos,
                                                               const float* __restrict__ rope_sin, const float* __restrict__ k_gate, HyRows r) {
    HY_PDL();
    const long long t = blockIdx.x;
    const int H = p.heads, D = p.dim, VD = p.vdim, half = p.rot_dims / 2, pos = p.rot_dims > 0 ? r.positions[t] : 0;
    const float sc = rsqrtf((float)D), qs = p.q_scaled ? sc : 1.f, ks = p.k_scaled ? sc : 1.f;
    const __nv_bfloat16* qr = q + t * ld; const __nv_bfloat16* kr = k + t * ld;
    const int nqk = H * D / 8, nv = H * VD / 8;
    for (int it = threadIdx.x; it < nqk + nv; it += blockDim.x) {
        if (it >= nqk) {
            const int i = (it - nqk) * 8; float f[8];
            unpack8(*reinterpret_cast<const uint4*>(v + t * ld + i), f);
            st8f(vv + t * H * VD + i, f);
            continue;
        }
        const int i = it * 8, d = i % D;
        float a[8], b[8];
        unpack8(*reinterpret_cast<const uint4*>(qr + i), a); unpack8(*reinterpret_cast<const uint4*>(kr + i), b);
        if (d < p.rot_dims) {
            const bool lo = d < half; const int j = lo ? d : d - half, o = lo ? i + half : i - half;
            float ao[8], bo[8], c[8], sn[8];
            unpack8(*reinterpret_cast<const uint4*>(qr + o), ao); unpack8(*reinterpret_cast<const uint4*>(kr + o), bo);
            ld8f(rope_cos + (long long)pos * half + j, c); ld8f(rope_sin + (long long)pos * half + j, sn);
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                a[e] = lo ? a[e] * c[e] - ao[e] * sn[e] : a[e] * c[e] + ao[e] * sn[e];
                b[e] = lo ? b[e] * c[e] - bo[e] * sn[e] : b[e] * c[e] + bo[e] * sn[e];
            }
        }
        const float kg = k_gate ? k_gate[t * H + i / D] : ks;
#pragma unroll
        for (int e = 0; e < 8; ++e) { a[e] *= qs; b[e] *= kg; }
        st8f(qq + t * H * D + i, a); st8f(kk + t * H * D + i, b);
        if (dec_channel) {
            float z[8]; ld8f(dec_channel + t * H * D + i, z);
#pragma unroll
            for (int e = 0; e < 8; ++e) z[e] = expf(log_sigmoidf_(z[e]) * inv_tau);
            st8f(dec_channel + t * H * D + i, z);
        }
    }
    if (dec_head) for (int i = threadIdx.x; i < H; i += blockDim.x) dec_head[t * H + i] = decay_head[i];
}
static bool lin_vec8_ok(bool f32, int dim, int vdim, int half, int ld, const void* q, const void* k, const void* v, const float* qq, const float* kk, const float* vv, const float* dec,
                        const float* rc, const float* rs) {
    auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    return !f32 && dim % 8 == 0 && vdim % 8 == 0 && half % 8 == 0 && ld % 8 == 0 && al(q) && al(k) && al(v) && al(qq) && al(kk) && al(vv) && al(dec) && al(rc) && al(rs);
}

// Gates of the matrix memory, one CTA per (sequence, head).  Every thread owns a run of consecutive rows.  Pass 1: log gates
// i = cap tanh(z_i / cap), f = logsigmoid(cap tanh(z_f / cap)) and the run's effect on the running maximum as a pair (A, B): m_out =
// max(m_in + A, B) with A = sum of f and B = the maximum reached from minus infinity (the update m <- max(m + f, i) composes that way).
// One thread chains the runs' pairs from the carried maximum; pass 2 walks each run again from its incoming maximum and writes
// dec = exp(f + m_(t-1) - m_t), gin = exp(i - m_t), floor_ = exp(-m_t).  The last row of a run takes the chained value as its maximum, so
// that the next run starts from exactly the number this one ended with: the maximum is only a stabiliser (state, normaliser and floor
// all carry exp(-m_t)), what matters is that every row divides by the same number the next row multiplies with.
constexpr int MLSTM_SCAN_THREADS = 128;
__global__ void __launch_bounds__(MLSTM_SCAN_THREADS) hy_mlstm_gates_kernel(const float* __restrict__ gates, int ldg, int H, float cap, float* __restrict__ mstate,
                                                                            float* __restrict__ dec, float* __restrict__ gin, float* __restrict__ floor_, HyRows r) {
    HY_PDL();
    __shared__ float sA[MLSTM_SCAN_THREADS], sB[MLSTM_SCAN_THREADS], sM[MLSTM_SCAN_THREADS + 1];
    const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int row0 = r.seq_row0[seq], len = r.seq_row0[seq + 1] - row0, pos0 = r.seq_pos0[seq];
    const int per = (len + MLSTM_SCAN_THREADS - 1) / MLSTM_SCAN_THREADS, t0 = min(len, tid * per), t1 = min(len, t0 + per);
    const float inv_cap = 1.0f / cap;
    float A = 0.f, B = -INFINITY;
    for (int t = t0; t < t1; ++t) {
        const long long row = row0 + t;
        const float i = cap * tanhf(gates[row * ldg + h] * inv_cap), f = log_sigmoidf_(cap * tanhf(gates[row * ldg + H + h] * inv_cap));
        gin[row * H + h] = i; dec[row * H + h] = f;
        A += f; B = fmaxf(B + f, i);
    }
    sA[tid] = A; sB[tid] = B;
    __syncthreads();
    if (tid == 0) {
        float* ms = mstate + (long long)r.seq_state[seq] * H + h;
        float m = pos0 > 0 ? *ms : 0.f;                    // a sequence that starts in this step starts from 0
        for (int j = 0; j < MLSTM_SCAN_THREADS; ++j) { sM[j] = m; m = fmaxf(m + sA[j], sB[j]); }
        sM[MLSTM_SCAN_THREADS] = m; *ms = m;
    }
    __syncthreads();
    float m = sM[tid];
    for (int t = t0; t < t1; ++t) {
        const long long at = (long long)(row0 + t) * H + h;
        const float f = dec[at], i = gin[at];
        const float mn = t == t1 - 1 ? sM[tid + 1] : fmaxf(f + m, i);
        dec[at] = expf(f + m - mn); gin[at] = expf(i - mn); floor_[at] = expf(-mn);
        m = mn;
    }
}
template <typename TA>
__global__ void __launch_bounds__(128) hy_mlstm_prep_kernel(int H, int D, int VD, const TA* __restrict__ q, const TA* __restrict__ k, const TA* __restrict__ v, int ld,
                                                            const float* __restrict__ gin, float* __restrict__ qq, float* __restrict__ kk, float* __restrict__ vv) {
    HY_PDL();
    const long long t = blockIdx.x;
    const float sc = rsqrtf((float)D);
    for (int i = threadIdx.x; i < H * D; i += blockDim.x) { qq[t * H * D + i] = ldf(q + t * ld + i) * sc; kk[t * H * D + i] = ldf(k + t * ld + i) * gin[t * H + i / D]; }
    for (int i = threadIdx.x; i < H * VD; i += blockDim.x) vv[t * H * VD + i] = ldf(v + t * ld + i);
}

// Operands of the recurrence that writes with the complement of its forget gate.  kk = 1 - f comes from sigmoid of the negated argument.
__device__ __forceinline__ void forget_gate(float z, float lower, float& f, float& w) {
    const float e = expf(-fabsf(z)), big = 1.0f / (1.0f + e), small = e * big, open = 1.0f - lower;      // sigmoid(|z|), sigmoid(-|z|)
    f = fmaf(open, z >= 0.f ? big : small, lower); w = open * (z >= 0.f ? small : big);
}
template <typename TA>
__global__ void __launch_bounds__(128) hy_forget_prep_kernel(int H, int D, int VD, const TA* __restrict__ q, const TA* __restrict__ z, const TA* __restrict__ v, int ld,
                                                             const float* __restrict__ bias, const float* __restrict__ lower, float* __restrict__ qq, float* __restrict__ kk,
                                                             float* __restrict__ vv, float* __restrict__ dec) {
    HY_PDL();
    const long long t = blockIdx.x;
    for (int i = threadIdx.x; i < H * D; i += blockDim.x) {
        float f, w; forget_gate(ldf(z + t * ld + i) + bias[i], lower[i], f, w);
        qq[t * H * D + i] = siluf_(ldf(q + t * ld + i)); dec[t * H * D + i] = f; kk[t * H * D + i] = w;
    }
    for (int i = threadIdx.x; i < H * VD; i += blockDim.x) vv[t * H * VD + i] = ldf(v + t * ld + i);
}
// The same for bf16 rows in aligned groups of 8 channels: 16 bytes per access, the same bits
__global__ void __launch_bounds__(128) hy_forget_prep_vec8_kernel(int nqk, int nv, const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ z,
                                                                  const __nv_bfloat16* __restrict__ v, int ld, const float* __restrict__ bias, const float* __restrict__ lower,
                                                                  float* __restrict__ qq, float* __restrict__ kk, float* __restrict__ vv, float* __restrict__ dec) {
    HY_PDL();
    const long long t = blockIdx.x;
    for (int it = threadIdx.x; it < (nqk + nv) / 8; it += blockDim.x) {
        float a[8];
        if (it * 8 >= nqk) {
            const int i = it * 8 - nqk;
            unpack8(*reinterpret_cast<const uint4*>(v + t * ld + i), a);
            st8f(vv + t * nv + i, a);
            continue;
        }
        const int i = it * 8;
        float b[8], lo[8], bi[8], f[8], w[8];
        unpack8(*reinterpret_cast<const uint4*>(q + t * ld + i), a); unpack8(*reinterpret_cast<const uint4*>(z + t * ld + i), b);
        ld8f(bias + i, bi); ld8f(lower + i, lo);
#pragma unroll
        for (int e = 0; e < 8; ++e) { a[e] = siluf_(a[e]); forget_gate(b[e] + bi[e], lo[e], f[e], w[e]); }
        st8f(qq + t * nqk + i, a); st8f(dec + t * nqk + i, f); st8f(kk + t * nqk + i, w);
    }
}

// The whole mixer between its two projections in one kernel (bf16; dim and vdim multiples of 8 up to 128), one CTA per (sequence, head), in two
// forms: token by token for decoding rows and portions of up to FW_FEW_ROWS rows, and block by block on the tensor cores for longer ones.  Both
// keep the fp32 state in registers for the whole portion, read the fused projection's rows by cp.async one block of FW_TB tokens ahead, and end
// with the RMS norm per head.
//
// Token by token: the block's gates are evaluated once into shared memory ([f | 1 - f | silu q] per token, fp32); the tokens then run one
// after the other without a barrier — a thread keeps DQ x 4 state rows of 8 value channels in registers (as pairs of rows for the
// packed fp32 multiply-adds), the 16 threads of a channel group meet in a reduce-scatter of shuffles per token — and the block's read-outs
// are RMS-normed per head and stored in the output projection's element type.  The order of every sum depends on the sizes alone, and a
// token's arithmetic does not depend on where in a block it falls.
constexpr int FW_TB = 16, FW_FEW_ROWS = HY_FORGET_FEW_ROWS;
__device__ __forceinline__ uint64_t pair2(float lo, float hi) { uint64_t r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ float2 unpair2(uint64_t p) { float2 r; asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(p)); return r; }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) { uint64_t r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) { uint64_t r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
template <int DQ>
__global__ void __launch_bounds__(256, 2) hy_forget_mix_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ z, const __nv_bfloat16* __restrict__ v, int ld,
                                                               const float* __restrict__ bias, const float* __restrict__ lower, const float* __restrict__ norm_w, float* __restrict__ state,
                                                               __nv_bfloat16* __restrict__ out, int ldo, int H, int D, int VD, float eps, HyRows r) {
    HY_PDL();
    constexpr int DP = 64 * DQ;                          // state rows padded to what the threads hold: f = 1, nothing written, nothing read
    extern __shared__ __align__(16) uint8_t fw_smem[];
    const int VP = (VD + 15) / 16 * 16, RAW = 2 * D + VD, nt = blockDim.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float* cv = reinterpret_cast<float*>(fw_smem);                       // [FW_TB][3][DP]
    float* os = cv + FW_TB * 3 * DP;                                     // [FW_TB][VP]
    __nv_bfloat16* raw = reinterpret_cast<__nv_bfloat16*>(os + FW_TB * VP);      // [2][FW_TB][q | z | v]
    const int seq = blockIdx.x, h = blockIdx.y;
    const long long row0 = r.seq_row0[seq]; const int len = r.seq_row0[seq + 1] - (int)row0, pos0 = r.seq_pos0[seq];
    if (len > FW_FEW_ROWS) return;                       // the block form takes this sequence
    q += row0 * ld + h * D; z += row0 * ld + h * D; v += row0 * ld + h * VD; out += row0 * ldo + h * VD;
    bias += h * D; lower += h * D;
    const int rl = lane >> 1, col0 = warp * 16 + (lane & 1) * 8;         // this thread: state rows j * 64 + rl * 4 .. + 3, value channels col0 .. + 7
    const bool col_ok = col0 < VD;
    auto fetch = [&](int b) {
        const int n = min(FW_TB, len - b * FW_TB) * (RAW / 8); __nv_bfloat16* dst = raw + (b & 1) * FW_TB * RAW;
        for (int i = tid; i < n; i += nt) {
            const int t = i / (RAW / 8), c = (i - t * (RAW / 8)) * 8; const long long at = (long long)(b * FW_TB + t) * ld;
            cp_async16(dst + t * RAW + c, c < D ? q + at + c : c < 2 * D ? z + at + (c - D) : v + at + (c - 2 * D));
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    float* st = state + (((long long)r.seq_state[seq] * H + h) * D) * VD + col0;
    uint64_t S[DQ][2][8];                                // [quad of rows][pair][value channel]
#pragma unroll
    for (int j = 0; j < DQ; ++j)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            float a[8], b[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) a[e] = b[e] = 0.f;
            const int d = j * 64 + rl * 4 + p * 2;       // D is even: both rows of a pair exist or neither does
            if (pos0 > 0 && col_ok && d < D) { ld8f(st + (long long)d * VD, a); ld8f(st + (long long)(d + 1) * VD, b); }
#pragma unroll
            for (int c = 0; c < 8; ++c) S[j][p][c] = pair2(a[c], b[c]);
        }
    for (int i = tid; i < FW_TB * (DP - D); i += nt) {   // padding rows
        float* row = cv + (i / (DP - D)) * 3 * DP + D + i % (DP - D);
        row[0] = 1.f; row[DP] = 0.f; row[2 * DP] = 0.f;
    }
    const int n_blocks = (len + FW_TB - 1) / FW_TB;
    for (int b = 0; b < n_blocks; ++b) {
        const int nb = min(FW_TB, len - b * FW_TB);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                 // block b has landed; everybody is done with block b - 1
        if (b + 1 < n_blocks) fetch(b + 1);
        const __nv_bfloat16* rb = raw + (b & 1) * FW_TB * RAW;
        for (int i = tid; i < nb * (D / 8); i += nt) {
            const int t = i / (D / 8), c = (i - t * (D / 8)) * 8;
            float a[8], g[8], lo[8], bi[8], f[8], w[8];
            unpack8(*reinterpret_cast<const uint4*>(rb + t * RAW + c), a); unpack8(*reinterpret_cast<const uint4*>(rb + t * RAW + D + c), g);
            ld8f(bias + c, bi); ld8f(lower + c, lo);
#pragma unroll
            for (int e = 0; e < 8; ++e) { a[e] = siluf_(a[e]); forget_gate(g[e] + bi[e], lo[e], f[e], w[e]); }
            float* row = cv + t * 3 * DP + c;
            st8f(row, f); st8f(row + DP, w); st8f(row + 2 * DP, a);
        }
        __syncthreads();
        if (warp * 16 < VD)
            for (int t = 0; t < nb; ++t) {
                const float* base = cv + t * 3 * DP + rl * 4;
                uint4 vr = make_uint4(0, 0, 0, 0);
                if (col_ok) vr = *reinterpret_cast<const uint4*>(rb + t * RAW + 2 * D + col0);
                float vf[8]; unpack8(vr, vf);
                uint64_t v2[8], o2[8];
#pragma unroll
                for (int c = 0; c < 8; ++c) { v2[c] = pair2(vf[c], vf[c]); o2[c] = 0ull; }
#pragma unroll
                for (int j = 0; j < DQ; ++j) {
                    const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(base + j * 64), w = *reinterpret_cast<const ulonglong2*>(base + DP + j * 64),
                                     qq = *reinterpret_cast<const ulonglong2*>(base + 2 * DP + j * 64);
#pragma unroll
                    for (int c = 0; c < 8; ++c) { S[j][0][c] = fma2(f.x, S[j][0][c], mul2(w.x, v2[c])); o2[c] = fma2(qq.x, S[j][0][c], o2[c]); }
#pragma unroll
                    for (int c = 0; c < 8; ++c) { S[j][1][c] = fma2(f.y, S[j][1][c], mul2(w.y, v2[c])); o2[c] = fma2(qq.y, S[j][1][c], o2[c]); }
                }
                float o[8];
#pragma unroll
                for (int c = 0; c < 8; ++c) { const float2 p = unpair2(o2[c]); o[c] = p.x + p.y; }
                // reduce-scatter over the 16 row lanes: bits 4, 3, 2 of the lane keep one of the 8 channels, bit 1 completes its sum
#pragma unroll
                for (int k = 4; k >= 1; k >>= 1) {
                    const int bit = k * 4; const bool up = lane & bit;
#pragma unroll
                    for (int c = 0; c < k; ++c) {
                        const float keep = up ? o[c + k] : o[c], give = up ? o[c] : o[c + k];
                        o[c] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
                    }
                }
                o[0] += __shfl_xor_sync(0xffffffffu, o[0], 2);
                if (!(lane & 2)) os[t * VP + col0 + ((lane >> 2) & 7)] = o[0];
            }
        __syncthreads();                                 // the block's read-outs are complete
        for (int t = warp; t < nb; t += nt >> 5) {
            float ss = 0.f;
            for (int c = lane; c < VD; c += 32) { const float x = os[t * VP + c]; ss = fmaf(x, x, ss); }
            const float rr = 1.0f / sqrtf(warp_sum(ss) / (float)VD + eps);
            for (int c = lane * 2; c < VD; c += 64)
                *reinterpret_cast<uint32_t*>(out + (long long)(b * FW_TB + t) * ldo + c) = pack_bf16x2(os[t * VP + c] * rr * norm_w[c], os[t * VP + c + 1] * rr * norm_w[c + 1]);
        }
    }
    if (!col_ok) return;
#pragma unroll
    for (int j = 0; j < DQ; ++j)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            const int d = j * 64 + rl * 4 + p * 2;
            if (d >= D) continue;
            float a[8], b[8];
#pragma unroll
            for (int c = 0; c < 8; ++c) { const float2 u = unpair2(S[j][p][c]); a[c] = u.x; b[c] = u.y; }
            st8f(st + (long long)d * VD, a); st8f(st + (long long)(d + 1) * VD, b);
        }
}

// Block by block: with B_t the product of the gates of a block's tokens up to t, o_t = (q_t B_t)^T S_in + sum over s <= t of A[t, s] v_s and
// S_out = diag(B_last) S_in + sum over s of (w_s prod over u > s of f_u) v_s^T, where w = 1 - f and A[t, s] = sum over channels of
// q_t w_s prod over s < u <= t of f_u.  Only products of gates appear, never a quotient: a gate may be as small as it likes.  Two of the sums
// are matrix products over the state (mma.sync m16n8k16, fp32 accumulation): a warp owns 16 value channels and holds S^T for them as
// accumulator fragments, which are the A operand of O^T = S^T (q B)^T as they stand; S^T += V^T (w ...) accumulates into them.  Operands that
// are not bfloat16 already (the state as read, q B, w times gates, A) enter as a bfloat16 value plus a bfloat16 remainder, so the products are
// accurate to about 2^-16 of their size (q B is rounded like the projection it comes from); the state itself stays fp32.  Tokens beyond the portion's end count as gates of one that write nothing.
template <int CV> __device__ __forceinline__ void load_cv(const float* p, float* f) {
#pragma unroll
    for (int e = 0; e < CV; e += 4) { const float4 x = *reinterpret_cast<const float4*>(p + e); f[e] = x.x; f[e + 1] = x.y; f[e + 2] = x.z; f[e + 3] = x.w; }
}
template <int CV> __device__ __forceinline__ void load_cv(const __nv_bfloat16* p, float* f) {
#pragma unroll
    for (int e = 0; e < CV; e += 4) { const uint2 x = *reinterpret_cast<const uint2*>(p + e); f[e] = bf16lo(x.x); f[e + 1] = bf16hi(x.x); f[e + 2] = bf16lo(x.y); f[e + 3] = bf16hi(x.y); }
}
template <int DP, int THREADS, int CTAS>      // CTAS per SM the registers are cut for: 2, or 1 where the grid does not fill the SMs once (the same arithmetic)
__global__ void __launch_bounds__(THREADS, CTAS) hy_forget_chunk_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ z, const __nv_bfloat16* __restrict__ v, int ld,
                                                                     const float* __restrict__ bias, const float* __restrict__ lower, const float* __restrict__ norm_w, float* __restrict__ state,
                                                                     __nv_bfloat16* __restrict__ out, int ldo, int H, int D, int VD, float eps, HyRows r) {
    HY_PDL();
    constexpr int TB = FW_TB, QP = DP + 8, AP = TB + 8, LG = DP / 4, NT = DP / 8, TPR = THREADS / TB, CV = DP / TPR < 8 ? DP / TPR : 8;      // TPR: threads per token in the row-wise phases
    extern __shared__ __align__(16) uint8_t fw_smem[];
    const int VP = (VD + 15) / 16 * 16, RP = 2 * D + VD + 8, OP = VP + 4, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, trow = tid / TPR, tsub = tid % TPR;
    float* fs = reinterpret_cast<float*>(fw_smem);                       // [TB][DP] gates
    float* ws = fs + TB * DP; float* qs = ws + TB * DP;                  // [TB][DP] 1 - gate, silu q
    float* bt = qs + TB * DP;                                            // [DP] product of the block's gates
    float* gb = bt + DP; float* gl = gb + DP;                            // [DP] gate biases and lower bounds of the head
    float* nw = gl + DP;                                                 // [VP] norm weights
    float* os = nw + VP;                                                 // [TB][OP] read-outs
    __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(os + TB * OP);  // [TB][QP] q B; w times the gates behind it (value, remainder)
    __nv_bfloat16 *kh = qh + TB * QP, *kl = kh + TB * QP;
    __nv_bfloat16 *ah = kl + TB * QP, *al = ah + TB * AP;                // [TB][AP] A (value, remainder)
    __nv_bfloat16* raw = al + TB * AP;                                   // [2][TB][q | z | v]
    const int seq = blockIdx.x, h = blockIdx.y;
    const long long row0 = r.seq_row0[seq]; const int len = r.seq_row0[seq + 1] - (int)row0, pos0 = r.seq_pos0[seq];
    if (len <= FW_FEW_ROWS) return;                      // the token-by-token form takes this sequence
    q += row0 * ld + h * D; z += row0 * ld + h * D; v += row0 * ld + h * VD; out += row0 * ldo + h * VD;
    const __nv_bfloat16 *qp = q + (long long)trow * ld + tsub * 8, *zp = z + (long long)trow * ld + tsub * 8, *vp = v + (long long)trow * ld + tsub * 8;      // this thread's pieces of the next block
    const long long block_step = (long long)TB * ld;
    auto fetch = [&](int b) {                            // called for b = 0, 1, 2, ...
        if (b * TB + trow < len) {
            __nv_bfloat16* dst = raw + ((b & 1) * TB + trow) * RP + tsub * 8;
#pragma unroll
            for (int k = 0; k < (DP + TPR * 8 - 1) / (TPR * 8); ++k)
                if ((tsub + k * TPR) * 8 < D) { cp_async16(dst + k * TPR * 8, qp + k * TPR * 8); cp_async16(dst + D + k * TPR * 8, zp + k * TPR * 8); }
            if (tsub * 8 < VD) cp_async16(dst + 2 * D, vp);        // 8 TPR >= VD
        }
        qp += block_step; zp += block_step; vp += block_step;
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const float inv_vd = 1.0f / (float)VD;
    fetch(0);
    for (int d = tid; d < DP; d += THREADS) { gb[d] = d < D ? bias[h * D + d] : 0.f; gl[d] = d < D ? lower[h * D + d] : 0.f; }
    for (int c = tid; c < VP; c += THREADS) nw[c] = c < VD ? norm_w[c] : 0.f;
    for (int i = tid; i < TB * AP; i += THREADS) ah[i] = al[i] = __float2bfloat16_rn(0.f);      // above the diagonal A stays zero
    // S^T fragments: tile n holds state rows d = n * 8 + (lane & 3) * 2, + 1 for the value channels v0, v0 + 8
    const int v0 = warp * 16 + (lane >> 2), dl = (lane & 3) * 2;
    float* st = state + (((long long)r.seq_state[seq] * H + h) * D) * VD;
    float S[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int d = n * 8 + dl + (c & 1), vc = v0 + (c >> 1) * 8;
            S[n][c] = (pos0 > 0 && d < D && vc < VD) ? st[(long long)d * VD + vc] : 0.f;
        }
    const int n_blocks = (len + TB - 1) / TB;
    for (int b = 0; b < n_blocks; ++b) {
        const int nb = min(TB, len - b * TB);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                 // block b has landed; everybody is done with block b - 1
        if (b + 1 < n_blocks) fetch(b + 1);
        __nv_bfloat16* rb = raw + (b & 1) * TB * RP;
#pragma unroll
        for (int k = 0; k < DP / CV / TPR; ++k) {        // gates and queries of one token, CV channels at a time
            const int c = (tsub + k * TPR) * CV; const bool live = trow < nb && c < D;
            float a[8], f[8], w[8];
            if (live) {
                float g[8], lo[8], bi[8];
                load_cv<CV>(rb + trow * RP + c, a); load_cv<CV>(rb + trow * RP + D + c, g); load_cv<CV>(gb + c, bi); load_cv<CV>(gl + c, lo);
#pragma unroll
                for (int e = 0; e < CV; ++e) {
                    a[e] = __fdividef(a[e], 1.0f + __expf(-a[e]));
                    const float x = g[e] + bi[e], ex = __expf(-fabsf(x)), big = __fdividef(1.0f, 1.0f + ex), small = ex * big, open = 1.0f - lo[e];
                    f[e] = fmaf(open, x >= 0.f ? big : small, lo[e]); w[e] = open * (x >= 0.f ? small : big);
                }
            } else {
#pragma unroll
                for (int e = 0; e < CV; ++e) { a[e] = 0.f; f[e] = 1.f; w[e] = 0.f; }
            }
#pragma unroll
            for (int e = 0; e < CV; e += 4) {
                *reinterpret_cast<float4*>(fs + trow * DP + c + e) = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
                *reinterpret_cast<float4*>(ws + trow * DP + c + e) = make_float4(w[e], w[e + 1], w[e + 2], w[e + 3]);
                *reinterpret_cast<float4*>(qs + trow * DP + c + e) = make_float4(a[e], a[e + 1], a[e + 2], a[e + 3]);
            }
        }
        if (trow >= nb) for (int c = tsub * 8; c < VD; c += TPR * 8) *reinterpret_cast<uint4*>(rb + trow * RP + 2 * D + c) = make_uint4(0, 0, 0, 0);
        __syncthreads();
        // q B forwards, w times the gates behind it backwards: one channel per thread
        for (int i = tid; i < 2 * DP; i += THREADS) {
            const int d = i % DP; const bool fwd = i < DP; const float* xs = (fwd ? qs : ws) + d;
            float p = 1.f;
#pragma unroll
            for (int t0 = 0; t0 < TB; t0 += 8) {         // eight tokens are read before their products are stored
                float g[8], x[8];
#pragma unroll
                for (int k = 0; k < 8; ++k) { const int t = fwd ? t0 + k : TB - 1 - t0 - k; g[k] = fs[t * DP + d]; x[k] = xs[t * DP]; }
#pragma unroll
                for (int k = 0; k < 8; ++k) {
                    const int t = fwd ? t0 + k : TB - 1 - t0 - k;
                    if (fwd) { p *= g[k]; qh[t * QP + d] = __float2bfloat16_rn(x[k] * p); }
                    else { split_bf16(x[k] * p, kh[t * QP + d], kl[t * QP + d]); p *= g[k]; }
                }
            }
            if (fwd) bt[d] = p;
        }
        // A: a group of LG lanes (four channels each; the last groups first, they had less to do above) walks column s = pi from its diagonal down (16 - pi rows), then column 15 - pi (pi + 1 rows): 17 steps
        for (int pi = THREADS / LG - 1 - tid / LG; pi < TB / 2; pi += THREADS / LG) {
            const int c = (lane % LG) * 4, turn = TB - pi;
            float acc[TB + 1];
            float4 g = *reinterpret_cast<const float4*>(ws + pi * DP + c);
            const float4 g2 = *reinterpret_cast<const float4*>(ws + (TB - 1 - pi) * DP + c);
#pragma unroll
            for (int k = 0; k <= TB; ++k) {
                const int t = k < turn ? pi + k : k - 1;
                const float4 qv = *reinterpret_cast<const float4*>(qs + t * DP + c), f = *reinterpret_cast<const float4*>(fs + t * DP + c);
                if (k > 0) {
                    const bool fresh = k == turn;
                    g.x = fresh ? g2.x : g.x * f.x; g.y = fresh ? g2.y : g.y * f.y; g.z = fresh ? g2.z : g.z * f.z; g.w = fresh ? g2.w : g.w * f.w;
                }
                acc[k] = fmaf(qv.x, g.x, qv.y * g.y) + fmaf(qv.z, g.z, qv.w * g.w);
            }
            // reduce-scatter over the group: a lane ends with one of the first 16 steps; the 17th is summed by all
            const unsigned mask = LG == 32 ? 0xffffffffu : 0xffffu << (lane & 16);
#pragma unroll
            for (int k = 8; k >= 1; k >>= 1) {
                const int bit = k * LG / TB; const bool up = lane & bit;
#pragma unroll
                for (int e = 0; e < k; ++e) { const float keep = up ? acc[e + k] : acc[e], give = up ? acc[e] : acc[e + k]; acc[e] = keep + __shfl_xor_sync(mask, give, bit); }
            }
            if (LG == 32) acc[0] += __shfl_xor_sync(mask, acc[0], 1);
#pragma unroll
            for (int o = LG / 2; o > 0; o >>= 1) acc[TB] += __shfl_xor_sync(mask, acc[TB], o);
            const int k = (lane % LG) / (LG / TB);
            if (LG == 16 || !(lane & 1)) { const int s = k < turn ? pi : TB - 1 - pi, t = k < turn ? pi + k : k - 1; split_bf16(acc[0], ah[t * AP + s], al[t * AP + s]); }
            if (lane % LG == 0) split_bf16(acc[TB], ah[(TB - 1) * AP + TB - 1 - pi], al[(TB - 1) * AP + TB - 1 - pi]);
        }
        __syncthreads();
        if (warp * 16 < VD) {
            float o[4][4];                               // [token half, and the same for the remainders]
#pragma unroll
            for (int e = 0; e < 4; ++e) o[0][e] = o[1][e] = o[2][e] = o[3][e] = 0.f;
            const int brow = (lane >> 4) * 8 + (lane & 7), bcol = ((lane >> 3) & 1) * 8;
            const uint32_t qha = smem_u32(qh + brow * QP + bcol);
#pragma unroll
            for (int ks = 0; ks < DP / 16; ++ks) {
                uint32_t sh[4], sl[4], b0, b1, b2, b3;
#pragma unroll
                for (int i = 0; i < 2; ++i) { split_pack(S[2 * ks + i][0], S[2 * ks + i][1], sh[2 * i], sl[2 * i]); split_pack(S[2 * ks + i][2], S[2 * ks + i][3], sh[2 * i + 1], sl[2 * i + 1]); }
                ldmatrix_x4(qha + ks * 32, b0, b1, b2, b3);
                mma_bf16_16816(o[0], sh[0], sh[1], sh[2], sh[3], b0, b1); mma_bf16_16816(o[1], sh[0], sh[1], sh[2], sh[3], b2, b3);
                mma_bf16_16816(o[2], sl[0], sl[1], sl[2], sl[3], b0, b1); mma_bf16_16816(o[3], sl[0], sl[1], sl[2], sl[3], b2, b3);
            }
            uint32_t va[4];                              // V^T of the warp's channels
            ldmatrix_x4_trans(smem_u32(rb + brow * RP + 2 * D + warp * 16 + bcol), va[0], va[1], va[2], va[3]);
            {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(smem_u32(ah + brow * AP + bcol), b0, b1, b2, b3);
                mma_bf16_16816(o[0], va[0], va[1], va[2], va[3], b0, b1); mma_bf16_16816(o[1], va[0], va[1], va[2], va[3], b2, b3);
                ldmatrix_x4(smem_u32(al + brow * AP + bcol), b0, b1, b2, b3);
                mma_bf16_16816(o[2], va[0], va[1], va[2], va[3], b0, b1); mma_bf16_16816(o[3], va[0], va[1], va[2], va[3], b2, b3);
            }
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) os[(j * 8 + dl + (e & 1)) * OP + v0 + (e >> 1) * 8] = o[j][e] + o[2 + j][e];
            const uint32_t kha = smem_u32(kh + (((lane >> 3) & 1) * 8 + (lane & 7)) * QP + (lane >> 4) * 8), kla = smem_u32(kl + (((lane >> 3) & 1) * 8 + (lane & 7)) * QP + (lane >> 4) * 8);
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                const float2 g0 = *reinterpret_cast<const float2*>(bt + n * 8 + dl), g1 = *reinterpret_cast<const float2*>(bt + n * 8 + 8 + dl);
                S[n][0] *= g0.x; S[n][1] *= g0.y; S[n][2] *= g0.x; S[n][3] *= g0.y;
                S[n + 1][0] *= g1.x; S[n + 1][1] *= g1.y; S[n + 1][2] *= g1.x; S[n + 1][3] *= g1.y;
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(kha + n * 16, b0, b1, b2, b3);
                mma_bf16_16816(S[n], va[0], va[1], va[2], va[3], b0, b1); mma_bf16_16816(S[n + 1], va[0], va[1], va[2], va[3], b2, b3);
                ldmatrix_x4_trans(kla + n * 16, b0, b1, b2, b3);
                mma_bf16_16816(S[n], va[0], va[1], va[2], va[3], b0, b1); mma_bf16_16816(S[n + 1], va[0], va[1], va[2], va[3], b2, b3);
            }
        }
        __syncthreads();                                 // the block's read-outs are complete
        {
            float x[8], wv[8], ss = 0.f;
            const bool mine = tsub * 8 < VD;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = 0.f;
            if (mine) { ld8f(os + trow * OP + tsub * 8, x); ld8f(nw + tsub * 8, wv); }
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(x[e], x[e], ss);
#pragma unroll
            for (int o = 1; o < TPR; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float rr = rsqrtf(fmaf(ss, inv_vd, eps));
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] *= rr * wv[e];
            if (mine && trow < nb)
                *reinterpret_cast<uint4*>(out + (long long)(b * TB + trow) * ldo + tsub * 8) = make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
        }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int d = n * 8 + dl + (c & 1), vc = v0 + (c >> 1) * 8;
            if (d < D && vc < VD) st[(long long)d * VD + vc] = S[n][c];
        }
}

// ---------------------------------------------------------------------------------------------------------------------------------
// router by table: one warp per token
// ---------------------------------------------------------------------------------------------------------------------------------
template <typename TA>
__global__ void __launch_bounds__(128) hy_moe_router_table_kernel(const int32_t* __restrict__ tokens, const int32_t* __restrict__ table, int vocab, int top, int shared,
                                                                  const TA* __restrict__ h, int ldh, const TA* __restrict__ w_sg, int W, int32_t* __restrict__ idx,
                                                                  float* __restrict__ wgt, int T) {
    HY_PDL();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp;
    if (t >= T) return;
    const int n = top + (shared >= 0 ? 1 : 0);
    int id = tokens[t]; id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    if (lane < top) { idx[(long long)t * n + lane] = table[(long long)id * top + lane]; wgt[(long long)t * n + lane] = 1.0f / (float)top; }
    if (shared >= 0) {
        float d = 0.f;
        for (int c = lane; c < W; c += 32) d = fmaf(ldf(h + (long long)t * ldh + c), ldf(w_sg + c), d);
        d = warp_sum(d);
        if (lane == 0) { idx[(long long)t * n + top] = shared; wgt[(long long)t * n + top] = sigmoidf_(d); }
    }
}

}  // namespace

cudaError_t hy_post_norm(bool f32, float* x, float beta, const float* y1, const float* rw1, const float* y2, const float* rw2, float branch_scale, const float* w, void* h, int ldh,
                         int T, int W, float eps, cudaStream_t s) {
    if (T <= 0) return cudaSuccess;
    if (rw1 && (!y1 || !y2 || !rw2)) return cudaErrorInvalidValue;
    auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (W % 4 == 0 && W <= 8192 && ldh % 4 == 0 && al(x) && al(y1) && al(y2) && al(rw1) && al(rw2) && al(w) && al(h))      // by the model's sizes alone, never by the step
    {
#define HY_PN(NV) (f32 ? launch_plain(hy_post_norm_reg_kernel<float, NV>, dim3(T), dim3(256), 0, s, x, beta, y1, rw1, y2, rw2, branch_scale, w, (float*)h, ldh, W, eps) \
                       : launch_plain(hy_post_norm_reg_kernel<__nv_bfloat16, NV>, dim3(T), dim3(256), 0, s, x, beta, y1, rw1, y2, rw2, branch_scale, w, (__nv_bfloat16*)h, ldh, W, eps))
        return W <= 1024 ? HY_PN(1) : W <= 2048 ? HY_PN(2) : W <= 4096 ? HY_PN(4) : HY_PN(8);
#undef HY_PN
    }
    return f32 ? launch_plain(hy_post_norm_kernel<float>, dim3(T), dim3(256), 0, s, x, beta, y1, rw1, y2, rw2, branch_scale, w, (float*)h, ldh, W, eps)
               : launch_plain(hy_post_norm_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, x, beta, y1, rw1, y2, rw2, branch_scale, w, (__nv_bfloat16*)h, ldh, W, eps);
}

cudaError_t hy_lin_prep(bool f32, const HyLinPrep& p, const void* q, const void* k, const void* v, int ld, float* qq, float* kk, float* vv, float* dec_channel, float tau,
                        const float* decay_head, float* dec_head, const float* rope_cos, const float* rope_sin, const HyRows& r, cudaStream_t s) {
    if (r.T <= 0) return cudaSuccess;
    if (p.rot_dims > 0 && (!rope_cos || !rope_sin || (p.rot_dims & 1) || p.rot_dims > p.dim)) return cudaErrorInvalidValue;
    using bf = __nv_bfloat16;
    if (lin_vec8_ok(f32, p.dim, p.vdim, p.rot_dims / 2, ld, q, k, v, qq, kk, vv, dec_channel, rope_cos, rope_sin))      // by the model's sizes alone
        return launch_plain(hy_lin_prep_vec8_kernel, dim3(r.T), dim3(128), 0, s, p, (const bf*)q, (const bf*)k, (const bf*)v, ld, qq, kk, vv, dec_channel, 1.0f / tau, decay_head,
                            dec_head, rope_cos, rope_sin, (const float*)nullptr, r);
    return f32 ? launch_plain(hy_lin_prep_kernel<float>, dim3(r.T), dim3(128), 0, s, p, (const float*)q, (const float*)k, (const float*)v, ld, qq, kk, vv, dec_channel, 1.0f / tau,
                              decay_head, dec_head, rope_cos, rope_sin, r)
               : launch_plain(hy_lin_prep_kernel<bf>, dim3(r.T), dim3(128), 0, s, p, (const bf*)q, (const bf*)k, (const bf*)v, ld, qq, kk, vv, dec_channel, 1.0f / tau, decay_head,
                              dec_head, rope_cos, rope_sin, r);
}

cudaError_t hy_forget_prep(bool f32, int heads, int dim, int vdim, const void* q, const void* z, const void* v, int ld, const float* bias, const float* lower, float* qq, float* kk, float* vv,
                           float* dec, int T, cudaStream_t s) {
    if (T <= 0) return cudaSuccess;
    using bf = __nv_bfloat16;
    if (heads * dim % 8 == 0 && heads * vdim % 8 == 0 && lin_vec8_ok(f32, 8, 8, 0, ld, q, z, v, qq, kk, vv, dec, bias, lower))      // by the model's sizes alone
        return launch_plain(hy_forget_prep_vec8_kernel, dim3(T), dim3(128), 0, s, heads * dim, heads * vdim, (const bf*)q, (const bf*)z, (const bf*)v, ld, bias, lower, qq, kk, vv, dec);
    return f32 ? launch_plain(hy_forget_prep_kernel<float>, dim3(T), dim3(128), 0, s, heads, dim, vdim, (const float*)q, (const float*)z, (const float*)v, ld, bias, lower, qq, kk, vv, dec)
               : launch_plain(hy_forget_prep_kernel<bf>, dim3(T), dim3(128), 0, s, heads, dim, vdim, (const bf*)q, (const bf*)z, (const bf*)v, ld, bias, lower, qq, kk, vv, dec);
}

bool hy_forget_mix_supported(int dim, int vdim) { return dim % 8 == 0 && vdim % 8 == 0 && dim >= 8 && vdim >= 8 && dim <= 128 && vdim <= 128; }
cudaError_t hy_forget_mix(int heads, int dim, int vdim, const void* q, const void* z, const void* v, int ld, const float* bias, const float* lower, const float* norm_w, float eps, float* state,
                          void* out, int ldo, bool few, bool many, const HyRows& r, cudaStream_t s) {
    if (r.T <= 0) return cudaSuccess;
    auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (!hy_forget_mix_supported(dim, vdim) || ld % 8 || ldo % 8 || !al(q) || !al(z) || !al(v) || !al(bias) || !al(lower) || !al(state) || !al(out)) return cudaErrorInvalidValue;
    using bf = __nv_bfloat16;
    const int dp = (dim + 63) / 64 * 64, vp = (vdim + 15) / 16 * 16;
    const size_t raw = (size_t)2 * FW_TB * (2 * dim + vdim + 8) * 2, smem_few = (size_t)FW_TB * (3 * dp + vp) * 4 + raw;
    const size_t smem_many = ((size_t)FW_TB * (3 * dp + vp + 4) + 3 * dp + vp) * 4 + (size_t)FW_TB * (3 * (dp + 8) + 2 * (FW_TB + 8)) * 2 + raw;
    const dim3 grid(r.S, heads);
    static bool done[7][16] = {};
    auto go = [&](auto kern, bool (&flag)[16], int threads, size_t smem) -> cudaError_t {
        if (cudaError_t e = ensure_dynamic_smem(kern, 100 * 1024, flag); e != cudaSuccess) return e;
        return launch_plain(kern, grid, dim3(threads), smem, s, (const bf*)q, (const bf*)z, (const bf*)v, ld, bias, lower, norm_w, state, (bf*)out, ldo, heads, dim, vdim, eps, r);
    };
    if (few) {           // a warp per 16 value channels
        const cudaError_t e = dp == 64 ? go(hy_forget_mix_kernel<1>, done[0], std::max(64, vp * 2), smem_few) : go(hy_forget_mix_kernel<2>, done[1], std::max(64, vp * 2), smem_few);
        if (e != cudaSuccess) return e;
    }
    if (many) {
        static int sms = 0;
        if (!sms) { int dev = 0; cudaGetDevice(&dev); if (cudaError_t e = cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev); e != cudaSuccess) return e; }
        // a token's 8-channel pieces are a power of two of threads
        const cudaError_t e = vp <= 64 ? (dp == 64 ? go(hy_forget_chunk_kernel<64, 128, 2>, done[2], 128, smem_many) : go(hy_forget_chunk_kernel<128, 128, 2>, done[3], 128, smem_many))
                                       : (dp == 64 ? go(hy_forget_chunk_kernel<64, 256, 2>, done[4], 256, smem_many) : r.S * heads <= sms ? go(hy_forget_chunk_kernel<128, 256, 1>, done[6], 256, smem_many) : go(hy_forget_chunk_kernel<128, 256, 2>, done[5], 256, smem_many));
        if (e != cudaSuccess) return e;
    }
    return cudaSuccess;
}

cudaError_t hy_mlstm_gates(const float* gates, int ldg, int heads, float cap, float* mstate, float* dec, float* gin, float* floor_, const HyRows& r, cudaStream_t s) {
    if (r.T <= 0) return cudaSuccess;
    return launch_plain(hy_mlstm_gates_kernel, dim3(r.S, heads), dim3(MLSTM_SCAN_THREADS), 0, s, gates, ldg, heads, cap, mstate, dec, gin, floor_, r);
}

cudaError_t hy_mlstm_prep(bool f32, int heads, int dim, int vdim, const void* q, const void* k, const void* v, int ld, const float* gin, float* qq, float* kk, float* vv, int T,
                          cudaStream_t s) {
    if (T <= 0) return cudaSuccess;
    using bf = __nv_bfloat16;
    if (lin_vec8_ok(f32, dim, vdim, 0, ld, q, k, v, qq, kk, vv, nullptr, nullptr, nullptr)) {
        HyRows r{}; r.T = T;                      // nothing is rotated: the kernel does not look at the rows' positions
        return launch_plain(hy_lin_prep_vec8_kernel, dim3(T), dim3(128), 0, s, HyLinPrep{heads, dim, vdim, true, false, 0}, (const bf*)q, (const bf*)k,
                            (const bf*)v, ld, qq, kk, vv, (float*)nullptr, 1.f, (const float*)nullptr, (float*)nullptr, (const float*)nullptr, (const float*)nullptr, gin, r);
    }
    return f32 ? launch_plain(hy_mlstm_prep_kernel<float>, dim3(T), dim3(128), 0, s, heads, dim, vdim, (const float*)q, (const float*)k, (const float*)v, ld, gin, qq, kk, vv)
               : launch_plain(hy_mlstm_prep_kernel<bf>, dim3(T), dim3(128), 0, s, heads, dim, vdim, (const bf*)q, (const bf*)k, (const bf*)v, ld, gin, qq, kk, vv);
}

cudaError_t hy_moe_router_table(bool f32, const int32_t* tokens, const int32_t* table, int vocab, int top, int shared, const void* h, int ldh, const void* w_sg, int W,
                                int32_t* idx, float* wgt, int T, cudaStream_t s) {
    if (T <= 0) return cudaSuccess;
    if (top < 1 || top + (shared >= 0 ? 1 : 0) > 32) return cudaErrorInvalidValue;
    using bf = __nv_bfloat16;
    return f32 ? launch_plain(hy_moe_router_table_kernel<float>, dim3((T + 3) / 4), dim3(128), 0, s, tokens, table, vocab, top, shared, (const float*)h, ldh, (const float*)w_sg, W, idx, wgt, T)
               : launch_plain(hy_moe_router_table_kernel<bf>, dim3((T + 3) / 4), dim3(128), 0, s, tokens, table, vocab, top, shared, (const bf*)h, ldh, (const bf*)w_sg, W, idx, wgt, T);
}

}  // namespace oa
