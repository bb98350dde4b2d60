// hybrid_blocks.cu — recurrences with one decay per head, bf16 (API: hybrid_kernels.hpp): lightning attention (S <- d S + k v^T) and the gated delta
// rule (S <- g S, u = beta (v - S^T k), S <- S + k u^T), each from the projections' rows to the heads' outputs in one kernel.
//
// Block form, one CTA per (sequence, head), blocks of 32 tokens.  With G_t the sum of the block's log decays up to t and e(t, s) = exp(G_t - G_s),
//   o_t   = exp(G_t) S_in^T q_t + sum over s <= t of e(t, s) (q_t . k_s) u_s
//   S_out = exp(G_last) S_in + sum over s of e(last, s) k_s u_s^T
// where u_s = v_s for lightning attention, and for the delta rule the u_s solve the unit lower triangular system
//   u_t + sum over s < t of beta_t e(t, s) (k_t . k_s) u_s = beta_t (v_t - exp(G_t) S_in^T k_t).
// The system is solved in two halves of 16 tokens: each half's 16 x 16 triangle is inverted (one column per lane), the second half's right side is
// corrected by the first half's solution.  Everything over the state or the values is a matrix product (mma.sync m16n8k16, fp32 accumulation): a
// warp owns 16 value channels and keeps S^T for them as accumulator fragments, which are the A operand of S^T k and S^T q as they stand; the
// right sides and the solutions pass from accumulator to operand in registers too.  k, q and v are bf16 rows (unit norms are factors on the
// products); every other operand enters as a bf16 value plus a bf16 remainder, so a product is accurate to about 2^-16 of its size, and the state
// itself stays fp32.  Only differences of log decays within a block are exponentiated, all of them <= 0.
//
// Token form (decoding rows, very short portions): one CTA per (sequence, head) loads the state once, a thread holds four value channels of every
// eighth row; the rows' partial sums meet in shared memory.  The order of every sum is fixed by the sizes.
#include <algorithm>

#include "hybrid_common.cuh"
#include "hybrid_kernels.hpp"

namespace oa {

namespace {

using namespace hyk;
using bf = __nv_bfloat16;
constexpr int BM_TB = 32, BM_FEW = HY_FORGET_FEW_ROWS;
constexpr float BM_LOG_MIN = -104.f;            // exp of it is zero in fp32: a stronger decay changes nothing

__device__ __forceinline__ float log_decay(float A_log, float x) { return fmaxf(-expf(A_log) * softplusf_(x), BM_LOG_MIN); }

struct BlockArgs {
    const bf *q, *k, *v; int ld; const bf *gate, *a, *b; int ld_in;
    const float *A_log, *dt_bias, *norm_w, *decay; float eps;
    float* state; void* out; int ldo, H, QH, D, VD;
};
constexpr int BM_PP = BM_TB + 8, BM_PM = BM_TB * BM_PP;      // pitch and size of a 32 x 32 matrix of bf16 operands
struct BlockSmem {          // offsets in bytes: three buffers of rows, read-outs, two sets of block matrices, triangles, two sets of factors per token, the norm's weight
    int QP, VP8, OP, row_bytes, buf, os, pm, lf, sc, nw, total;
    __host__ __device__ BlockSmem(bool delta, int DP, int VP) {
        QP = DP + 8; VP8 = VP + 8; OP = VP + 4;
        row_bytes = (2 * QP + (delta ? 2 : 1) * VP8) * 2; buf = BM_TB * row_bytes;
        os = 3 * buf; pm = os + BM_TB * OP * 4; lf = pm + 2 * 4 * BM_PM * 2; sc = lf + BM_TB * 20 * 4; nw = sc + (2 * 6 * BM_TB + 2 * BM_TB) * 4; total = nw + VP * 4;
    }
};

// A block passes through three stages, each a block ahead of the next: its rows arrive (cp.async), the factors per token and the products of its rows with
// one another are made, it meets the state.  Per block there are two barriers: between A and B the state's products of block b beside the row products
// of block b + 1, between B and A the read-outs of block b beside the triangles of block b + 1 and the factors of block b + 2.
template <bool DELTA, int DP, int THREADS>
__global__ void __launch_bounds__(THREADS, THREADS == 128 ? 2 : 1) hy_block_memory_kernel(BlockArgs p, HyRows r) {
    HY_PDL();
    constexpr int NW = THREADS / 32, TPR = THREADS / BM_TB, NT = DP / 8, PP = BM_PP;
    extern __shared__ __align__(16) uint8_t bm_smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, seq = blockIdx.x, h = blockIdx.y, D = p.D, VD = p.VD, VP = (VD + 15) / 16 * 16;
    const long long row0 = r.seq_row0[seq]; const int len = r.seq_row0[seq + 1] - (int)row0, pos0 = r.seq_pos0[seq];
    if (len <= BM_FEW) return;                           // the token form takes this sequence
    const BlockSmem L(DELTA, DP, VP);
    const int QP = L.QP, VP8 = L.VP8, OP = L.OP;
    float* os = reinterpret_cast<float*>(bm_smem + L.os);            // [32][OP] read-outs
    float* lf = reinterpret_cast<float*>(bm_smem + L.lf);            // [32][20] the triangles' entries below the diagonal, column s of a triangle in row s
    float* sc = reinterpret_cast<float*>(bm_smem + L.sc);
    float* pw = sc + 12 * BM_TB;                                     // powers of a fixed decay
    const int qh = h / (p.H / p.QH), trow = tid / TPR, tsub = tid % TPR;
    const bf* qg = p.q + row0 * p.ld + (long long)qh * D; const bf* kg = p.k + row0 * p.ld + (long long)qh * D; const bf* vg = p.v + row0 * p.ld + (long long)h * VD;
    const bf* gg = DELTA ? p.gate + row0 * p.ld_in + (long long)h * VD : nullptr;
    const int n_blocks = (len + BM_TB - 1) / BM_TB;
    auto Qs = [&](int b) { return reinterpret_cast<bf*>(bm_smem + (b % 3) * L.buf); };
    auto Ks = [&](int b) { return Qs(b) + BM_TB * QP; };
    auto Vs = [&](int b) { return Qs(b) + 2 * BM_TB * QP; };
    auto Gt = [&](int b) { return Qs(b) + 2 * BM_TB * QP + BM_TB * VP8; };
    // block matrices, each a value and a remainder [32][PP]: ph | pl e(t, s) q_t . k_s; mh | ml inverted triangles on the diagonal, the negated block below
    auto ph_of = [&](int b) { return reinterpret_cast<bf*>(bm_smem + L.pm) + (b & 1) * 4 * BM_PM; };
    auto mh_of = [&](int b) { return ph_of(b) + 2 * BM_PM; };
    // factors per token: of q and of k, G, exp(G), e(last, s), beta
    struct Factors { float *rq, *rk, *Gs, *eG, *wl, *bt; };
    auto factors_of = [&](int b) { float* f = sc + (b & 1) * 6 * BM_TB; return Factors{f, f + BM_TB, f + 2 * BM_TB, f + 3 * BM_TB, f + 4 * BM_TB, f + 5 * BM_TB}; };
    for (int i = tid; i < 3 * L.buf / 16; i += THREADS) reinterpret_cast<uint4*>(bm_smem)[i] = make_uint4(0, 0, 0, 0);      // padding columns, and rows no block has filled yet
    for (int i = tid; i < 8 * BM_PM * 2 / 16; i += THREADS) reinterpret_cast<uint4*>(bm_smem + L.pm)[i] = make_uint4(0, 0, 0, 0);      // above the diagonal the matrices stay zero
    bf a_next = __float2bfloat16_rn(0.f), b_next = a_next;
    constexpr int QN = DP / 8 / TPR;                     // this thread's 16-byte pieces of a row of q and of k; of v and the gate: two
    const long long step = (long long)BM_TB * p.ld, step_in = (long long)BM_TB * p.ld_in;
    const bf *qp = qg + (long long)trow * p.ld + tsub * 8, *kp = kg + (long long)trow * p.ld + tsub * 8, *vp = vg + (long long)trow * p.ld + tsub * 8;
    const bf *gp = DELTA ? gg + (long long)trow * p.ld_in + tsub * 8 : nullptr, *ap = DELTA ? p.a + (row0 + lane) * p.ld_in + h : nullptr, *bp = DELTA ? p.b + (row0 + lane) * p.ld_in + h : nullptr;
    auto fetch = [&](int b) {                            // called for b = 0, 1, 2, ...: TPR threads per token, 16 bytes per access
        if (b * BM_TB + trow < len) {
            bf* qd = Qs(b) + trow * QP + tsub * 8; bf* vd = Vs(b) + trow * VP8 + tsub * 8;
#pragma unroll
            for (int i = 0; i < QN; ++i)
                if ((tsub + i * TPR) * 8 < D) { cp_async16(qd + i * TPR * 8, qp + i * TPR * 8); cp_async16(qd + BM_TB * QP + i * TPR * 8, kp + i * TPR * 8); }
#pragma unroll
            for (int i = 0; i < 2; ++i)
                if ((tsub + i * TPR) * 8 < VD) { cp_async16(vd + i * TPR * 8, vp + i * TPR * 8); if (DELTA) cp_async16(vd + BM_TB * VP8 + i * TPR * 8, gp + i * TPR * 8); }
        }
        if (DELTA && warp == 0 && b * BM_TB + lane < len) { a_next = *ap; b_next = *bp; }
        qp += step; kp += step; vp += step;
        if (DELTA) { gp += step_in; ap += step_in; bp += step_in; }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const float al = DELTA ? p.A_log[h] : 0.f, db = DELTA ? p.dt_bias[h] : 0.f, qscale = rsqrtf((float)D);
    const int brow = (lane >> 4) * 8 + (lane & 7), bcol = ((lane >> 3) & 1) * 8, dl = (lane & 3) * 2;      // ldmatrix lane addresses of a B operand of 16 rows x 16 columns
    auto make_factors = [&](int b) {
        const int nb = min(BM_TB, len - b * BM_TB); const Factors f = factors_of(b);
        if (DELTA) {
            const bf *Qb = Qs(b), *Kb = Ks(b);
            float sq = 0.f, sk = 0.f;
#pragma unroll
            for (int i = 0; i < QN; ++i) {               // padding columns are zero
                const int c = (tsub + i * TPR) * 8;
                float x[8], y[8];
                unpack8(*reinterpret_cast<const uint4*>(Qb + trow * QP + c), x); unpack8(*reinterpret_cast<const uint4*>(Kb + trow * QP + c), y);
                sq += ((x[0] * x[0] + x[1] * x[1]) + (x[2] * x[2] + x[3] * x[3])) + ((x[4] * x[4] + x[5] * x[5]) + (x[6] * x[6] + x[7] * x[7]));
                sk += ((y[0] * y[0] + y[1] * y[1]) + (y[2] * y[2] + y[3] * y[3])) + ((y[4] * y[4] + y[5] * y[5]) + (y[6] * y[6] + y[7] * y[7]));
            }
#pragma unroll
            for (int o = 1; o < TPR; o <<= 1) { sq += __shfl_xor_sync(0xffffffffu, sq, o); sk += __shfl_xor_sync(0xffffffffu, sk, o); }
            if (tsub == 0) { f.rq[trow] = qscale * rsqrtf(sq + 1e-6f); f.rk[trow] = rsqrtf(sk + 1e-6f); }
            if (warp == 0) {                             // lane = token
                float G = lane < nb ? log_decay(al, ldf(&a_next) + db) : 0.f;
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) { const float u = __shfl_up_sync(0xffffffffu, G, o); if (lane >= o) G += u; }
                const float Gl = __shfl_sync(0xffffffffu, G, 31);
                f.Gs[lane] = G; f.eG[lane] = expf(G); f.wl[lane] = lane < nb ? expf(Gl - G) : 0.f; f.bt[lane] = lane < nb ? sigmoidf_(ldf(&b_next)) : 0.f;
            }
        } else if (tid < BM_TB) { f.rq[tid] = f.rk[tid] = 1.f; f.eG[tid] = pw[tid + 1]; f.wl[tid] = tid < nb ? pw[nb - 1 - tid] : 0.f; }
    };
    // products of a block's rows with one another: units of 16 x 16, the diagonal ones and the one below
    auto row_products = [&](int b) {
        const bf *Qb = Qs(b), *Kb = Ks(b); const Factors f = factors_of(b); bf *ph = ph_of(b), *mh = mh_of(b);
        for (int u = warp; u < (DELTA ? 6 : 3); u += NW) {
            const bool kk = u >= 3; const int m = (u % 3 + 1) / 2, np = u % 3 == 2 ? 1 : 0;      // (0, 0), (1, 0), (1, 1)
            float acc[2][4] = {};
            const uint32_t aa = smem_u32((kk ? Kb : Qb) + (m * 16 + (lane & 15)) * QP + (lane >> 4) * 8), ba = smem_u32(Kb + (np * 16 + brow) * QP + bcol);
#pragma unroll
            for (int ks = 0; ks < DP / 16; ++ks) {
                uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
                ldmatrix_x4(aa + ks * 32, a0, a1, a2, a3); ldmatrix_x4(ba + ks * 32, b0, b1, b2, b3);
                mma_bf16_16816(acc[0], a0, a1, a2, a3, b0, b1); mma_bf16_16816(acc[1], a0, a1, a2, a3, b2, b3);
            }
            // this thread's rows t and columns s, s + 1: their factors first, then the eight entries, stored in pairs
            const int t0 = m * 16 + (lane >> 2), s0 = np * 16 + dl;
            float ct[2], gt[2], cs[2][2], gs[2][2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int t = t0 + i * 8;
                ct[i] = kk ? f.rk[t] * f.bt[t] : f.rq[t]; gt[i] = DELTA ? f.Gs[t] : 0.f;
#pragma unroll
                for (int k = 0; k < 2; ++k) { cs[i][k] = f.rk[s0 + i * 8 + k]; gs[i][k] = DELTA ? f.Gs[s0 + i * 8 + k] : 0.f; }
            }
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int t = t0 + i * 8, s = s0 + j * 8;
                    float x[2];
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        const bool live = kk ? s + k < t : s + k <= t;
                        x[k] = live ? acc[j][i * 2 + k] * ct[i] * cs[j][k] * (DELTA ? __expf(gt[i] - gs[j][k]) : pw[t - s - k]) : 0.f;
                    }
                    if (kk && m == np) { lf[(m * 16 + s - np * 16) * 20 + t - m * 16] = x[0]; lf[(m * 16 + s + 1 - np * 16) * 20 + t - m * 16] = x[1]; }      // column by column
                    else {
                        uint32_t hi, lo; split_pack(kk ? -x[0] : x[0], kk ? -x[1] : x[1], hi, lo);
                        bf* d = (kk ? mh : ph) + t * PP + s;
                        *reinterpret_cast<uint32_t*>(d) = hi; *reinterpret_cast<uint32_t*>(d + BM_PM) = lo;
                    }
                }
        }
    };
    auto invert = [&](int b) {                           // one warp: column lane & 15 of the inverse of triangle lane >> 4
        bf* mh = mh_of(b);
        const float* lr = lf + (lane >> 4) * 16 * 20; const int c = lane & 15, t0 = (lane >> 4) * 16;
        float x[16];
#pragma unroll
        for (int t = 0; t < 16; ++t) x[t] = t == c ? 1.f : 0.f;
#pragma unroll
        for (int s = 0; s < 15; ++s)                     // x[s] is final: take it off the rows below
#pragma unroll
            for (int q = (s + 1) / 4; q < 4; ++q) {
                const float4 l4 = *reinterpret_cast<const float4*>(lr + s * 20 + q * 4);
                if (4 * q > s) x[4 * q] = fmaf(-l4.x, x[s], x[4 * q]);
                if (4 * q + 1 > s) x[4 * q + 1] = fmaf(-l4.y, x[s], x[4 * q + 1]);
                if (4 * q + 2 > s) x[4 * q + 2] = fmaf(-l4.z, x[s], x[4 * q + 2]);
                if (4 * q + 3 > s) x[4 * q + 3] = fmaf(-l4.w, x[s], x[4 * q + 3]);
            }
#pragma unroll
        for (int t = 0; t < 16; ++t) split_bf16(x[t], mh[(t0 + t) * PP + t0 + c], mh[BM_PM + (t0 + t) * PP + t0 + c]);
    };
    float* nw = reinterpret_cast<float*>(bm_smem + L.nw);
    if (DELTA) for (int i = tid; i < VD; i += THREADS) nw[i] = p.norm_w[i];
    if (!DELTA && tid == 0) { const float d = p.decay[h]; float x = 1.f; for (int i = 0; i <= BM_TB; ++i) { pw[i] = x; x *= d; } }
    __syncthreads();                                     // the buffers are cleared
    fetch(0);
    // S^T fragments: tile n holds state rows n * 8 + (lane & 3) * 2, + 1 for the value channels v0, v0 + 8
    const int v0 = warp * 16 + (lane >> 2); const bool mine = warp * 16 < VD;
    float* st = p.state + (((long long)r.seq_state[seq] * p.H + h) * D) * VD;
    float S[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int d = n * 8 + dl + (c & 1), vc = v0 + (c >> 1) * 8;
            S[n][c] = (pos0 > 0 && d < D && vc < VD) ? st[(long long)d * VD + vc] : 0.f;
        }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    make_factors(0);
    if (n_blocks > 1) fetch(1);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    row_products(0);
    __syncthreads();
    if (DELTA && warp == NW - 1) invert(0);
    if (n_blocks > 1) make_factors(1);
    for (int b = 0; b < n_blocks; ++b) {
        const int nb = min(BM_TB, len - b * BM_TB);
        __syncthreads();                                 // A: matrices of block b, factors of block b + 1; everybody is done with block b - 1
        if (b + 2 < n_blocks) fetch(b + 2);
        if (b + 1 < n_blocks) row_products(b + 1);
        const bf *Qb = Qs(b), *Kb = Ks(b), *Vb = Vs(b), *ph = ph_of(b), *pl = ph + BM_PM, *mh = mh_of(b), *ml = mh + BM_PM;
        const Factors fc = factors_of(b); const float *rq = fc.rq, *rk = fc.rk, *eG = fc.eG, *wl = fc.wl, *bt = fc.bt;
        float kS[4][4] = {}, qS[4][4] = {};              // S^T k and S^T q of the warp's channels: [token tile][..]
        if (mine) {
            const uint32_t ka = smem_u32(Kb + brow * QP + bcol), qa = smem_u32(Qb + brow * QP + bcol);
#pragma unroll
            for (int ks = 0; ks < DP / 16; ++ks) {
                uint32_t sh[4], sl[4], kf[2][4], qf[2][4];
#pragma unroll
                for (int g = 0; g < 2; ++g) {
                    if (DELTA) ldmatrix_x4(ka + (g * 16 * QP + ks * 16) * 2, kf[g][0], kf[g][1], kf[g][2], kf[g][3]);
                    ldmatrix_x4(qa + (g * 16 * QP + ks * 16) * 2, qf[g][0], qf[g][1], qf[g][2], qf[g][3]);
                }
#pragma unroll
                for (int i = 0; i < 2; ++i) { split_pack(S[2 * ks + i][0], S[2 * ks + i][1], sh[2 * i], sl[2 * i]); split_pack(S[2 * ks + i][2], S[2 * ks + i][3], sh[2 * i + 1], sl[2 * i + 1]); }
                auto pass = [&](const uint32_t (&x)[4]) {        // an accumulator's two products lie a whole pass apart
#pragma unroll
                    for (int g = 0; g < 2; ++g) {
                        if (DELTA) { mma_bf16_16816(kS[2 * g], x[0], x[1], x[2], x[3], kf[g][0], kf[g][1]); mma_bf16_16816(kS[2 * g + 1], x[0], x[1], x[2], x[3], kf[g][2], kf[g][3]); }
                        mma_bf16_16816(qS[2 * g], x[0], x[1], x[2], x[3], qf[g][0], qf[g][1]); mma_bf16_16816(qS[2 * g + 1], x[0], x[1], x[2], x[3], qf[g][2], qf[g][3]);
                    }
                };
                pass(sh); pass(sl);
            }
        }
        if (mine) {
            // tokens of an accumulator tile n: n * 8 + dl, + 1; of an A operand half g: the tiles 2 g, 2 g + 1
            uint32_t va[2][4];                           // V^T of the warp's channels, in the accumulators' layout
#pragma unroll
            for (int g = 0; g < 2; ++g) ldmatrix_x4_trans(smem_u32(Vb + (g * 16 + brow) * VP8 + warp * 16 + bcol), va[g][0], va[g][1], va[g][2], va[g][3]);
            const uint32_t mha = smem_u32(mh + brow * PP + bcol), mla = smem_u32(ml + brow * PP + bcol), pha = smem_u32(ph + brow * PP + bcol), pla = smem_u32(pl + brow * PP + bcol);
            float U[4][4]; uint32_t uh[2][4], ul[2][4];
            auto times = [&](float (&x)[4], float (&y)[4], const uint32_t (&ah)[4], const uint32_t (&alo)[4], uint32_t hi, uint32_t lo, bool rem) {      // (ah + alo) . (hi + lo)^T of one 16 x 16 block, onto two tiles
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(hi, b0, b1, b2, b3);
                mma_bf16_16816(x, ah[0], ah[1], ah[2], ah[3], b0, b1); mma_bf16_16816(y, ah[0], ah[1], ah[2], ah[3], b2, b3);
                if (rem) { mma_bf16_16816(x, alo[0], alo[1], alo[2], alo[3], b0, b1); mma_bf16_16816(y, alo[0], alo[1], alo[2], alo[3], b2, b3); }
                ldmatrix_x4(lo, b0, b1, b2, b3);
                mma_bf16_16816(x, ah[0], ah[1], ah[2], ah[3], b0, b1); mma_bf16_16816(y, ah[0], ah[1], ah[2], ah[3], b2, b3);
            };
            auto blk = [&](int tg, int sg) -> uint32_t { return (uint32_t)(tg * 16 * PP + sg * 16) * 2; };
            if (DELTA) {
                float X[4][4];
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    const int t = n * 8 + dl;
                    const float f0 = eG[t] * rk[t], f1 = eG[t + 1] * rk[t + 1], b0 = bt[t], b1 = bt[t + 1];
                    const uint32_t vlo = va[n >> 1][(n & 1) * 2], vhi = va[n >> 1][(n & 1) * 2 + 1];
                    X[n][0] = b0 * (bf16lo(vlo) - f0 * kS[n][0]); X[n][1] = b1 * (bf16hi(vlo) - f1 * kS[n][1]);
                    X[n][2] = b0 * (bf16lo(vhi) - f0 * kS[n][2]); X[n][3] = b1 * (bf16hi(vhi) - f1 * kS[n][3]);
                }
#pragma unroll
                for (int g = 0; g < 2; ++g) {
                    uint32_t xh[4], xl[4];
                    if (g == 1) times(X[2], X[3], uh[0], ul[0], mha + blk(1, 0), mla + blk(1, 0), true);
#pragma unroll
                    for (int i = 0; i < 2; ++i) { split_pack(X[2 * g + i][0], X[2 * g + i][1], xh[2 * i], xl[2 * i]); split_pack(X[2 * g + i][2], X[2 * g + i][3], xh[2 * i + 1], xl[2 * i + 1]); }
#pragma unroll
                    for (int e = 0; e < 4; ++e) U[2 * g][e] = U[2 * g + 1][e] = 0.f;
                    times(U[2 * g], U[2 * g + 1], xh, xl, mha + blk(g, g), mla + blk(g, g), true);
#pragma unroll
                    for (int i = 0; i < 2; ++i) { split_pack(U[2 * g + i][0], U[2 * g + i][1], uh[g][2 * i], ul[g][2 * i]); split_pack(U[2 * g + i][2], U[2 * g + i][3], uh[g][2 * i + 1], ul[g][2 * i + 1]); }
                }
            } else {
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    const uint32_t vlo = va[n >> 1][(n & 1) * 2], vhi = va[n >> 1][(n & 1) * 2 + 1];
                    U[n][0] = bf16lo(vlo); U[n][1] = bf16hi(vlo); U[n][2] = bf16lo(vhi); U[n][3] = bf16hi(vhi);
                }
#pragma unroll
                for (int g = 0; g < 2; ++g)
#pragma unroll
                    for (int e = 0; e < 4; ++e) { uh[g][e] = va[g][e]; ul[g][e] = 0u; }
            }
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                const int t = n * 8 + dl; const float f0 = eG[t] * rq[t], f1 = eG[t + 1] * rq[t + 1];
                qS[n][0] *= f0; qS[n][1] *= f1; qS[n][2] *= f0; qS[n][3] *= f1;
            }
            {
                const int tg[3] = {0, 1, 1}, sg[3] = {0, 0, 1};
                uint32_t f[3][4];
                auto pass = [&](const uint32_t (&x)[2][4]) {
#pragma unroll
                    for (int i = 0; i < 3; ++i) {
                        mma_bf16_16816(qS[2 * tg[i]], x[sg[i]][0], x[sg[i]][1], x[sg[i]][2], x[sg[i]][3], f[i][0], f[i][1]);
                        mma_bf16_16816(qS[2 * tg[i] + 1], x[sg[i]][0], x[sg[i]][1], x[sg[i]][2], x[sg[i]][3], f[i][2], f[i][3]);
                    }
                };
#pragma unroll
                for (int i = 0; i < 3; ++i) ldmatrix_x4(pha + blk(tg[i], sg[i]), f[i][0], f[i][1], f[i][2], f[i][3]);
                pass(uh);
                if (DELTA) pass(ul);
#pragma unroll
                for (int i = 0; i < 3; ++i) ldmatrix_x4(pla + blk(tg[i], sg[i]), f[i][0], f[i][1], f[i][2], f[i][3]);
                pass(uh);
            }
#pragma unroll
            for (int n = 0; n < 4; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) os[(n * 8 + dl + (e & 1)) * OP + v0 + (e >> 1) * 8] = qS[n][e];
            // S^T <- exp(G_last) S^T + (U e(last, .))^T K
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                const int t = n * 8 + dl; const float f0 = wl[t] * rk[t], f1 = wl[t + 1] * rk[t + 1];
                U[n][0] *= f0; U[n][1] *= f1; U[n][2] *= f0; U[n][3] *= f1;
            }
#pragma unroll
            for (int g = 0; g < 2; ++g)
#pragma unroll
                for (int i = 0; i < 2; ++i) { split_pack(U[2 * g + i][0], U[2 * g + i][1], uh[g][2 * i], ul[g][2 * i]); split_pack(U[2 * g + i][2], U[2 * g + i][3], uh[g][2 * i + 1], ul[g][2 * i + 1]); }
            const float fS = DELTA ? eG[BM_TB - 1] : pw[nb];
            const uint32_t kt = smem_u32(Kb + (((lane >> 3) & 1) * 8 + (lane & 7)) * QP + (lane >> 4) * 8);
#pragma unroll
            for (int n = 0; n < NT; n += 4) {            // four tiles of state rows at a time: an accumulator's four products lie four apart
                uint32_t f[2][2][4];
#pragma unroll
                for (int g = 0; g < 2; ++g)
#pragma unroll
                    for (int j = 0; j < 2; ++j) ldmatrix_x4_trans(kt + (g * 16 * QP + (n + 2 * j) * 8) * 2, f[g][j][0], f[g][j][1], f[g][j][2], f[g][j][3]);
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) S[n + j][e] *= fS;
#pragma unroll
                for (int g = 0; g < 2; ++g) {
#pragma unroll
                    for (int j = 0; j < 4; ++j) mma_bf16_16816(S[n + j], uh[g][0], uh[g][1], uh[g][2], uh[g][3], f[g][j >> 1][(j & 1) * 2], f[g][j >> 1][(j & 1) * 2 + 1]);
#pragma unroll
                    for (int j = 0; j < 4; ++j) mma_bf16_16816(S[n + j], ul[g][0], ul[g][1], ul[g][2], ul[g][3], f[g][j >> 1][(j & 1) * 2], f[g][j >> 1][(j & 1) * 2 + 1]);
                }
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                 // B: read-outs of block b, triangles of block b + 1, rows of block b + 2
        if (DELTA && warp == NW - 1 && b + 1 < n_blocks) invert(b + 1);
        if (b + 2 < n_blocks) make_factors(b + 2);
        const long long trow_g = row0 + b * BM_TB + trow;
        if (DELTA) {
            float x[2][8], ss = 0.f;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int c = (tsub + k * TPR) * 8;
                if (c < VD) {
                    ld8f(os + trow * OP + c, x[k]);
#pragma unroll
                    for (int e = 0; e < 8; ++e) ss = fmaf(x[k][e], x[k][e], ss);
                }
            }
#pragma unroll
            for (int o = 1; o < TPR; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float rr = rsqrtf(ss / (float)VD + p.eps);
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int c = (tsub + k * TPR) * 8;
                if (c < VD && trow < nb) {
                    float g[8], w[8];
                    unpack8(*reinterpret_cast<const uint4*>(Gt(b) + trow * VP8 + c), g); ld8f(nw + c, w);
#pragma unroll
                    for (int e = 0; e < 8; ++e) x[k][e] *= rr * w[e] * silu_fast_f32(g[e]);
                    *reinterpret_cast<uint4*>(reinterpret_cast<bf*>(p.out) + trow_g * p.ldo + (long long)h * VD + c) =
                        make_uint4(pack_bf16x2(x[k][0], x[k][1]), pack_bf16x2(x[k][2], x[k][3]), pack_bf16x2(x[k][4], x[k][5]), pack_bf16x2(x[k][6], x[k][7]));
                }
            }
        } else if (trow < nb)
            for (int c = tsub * 4; c < VD; c += TPR * 4)
                *reinterpret_cast<float4*>(reinterpret_cast<float*>(p.out) + trow_g * p.ldo + (long long)h * VD + c) = *reinterpret_cast<const float4*>(os + trow * OP + c);
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int d = n * 8 + dl + (c & 1), vc = v0 + (c >> 1) * 8;
            if (d < D && vc < VD) st[(long long)d * VD + vc] = S[n][c];
        }
}

// ---- token form ----
struct FewArgs {
    BlockArgs p;
    const bf* in; const float* conv_w; int taps, C; const bf* tails;      // delta rule: the short convolution's input rows [T, ld_in] of C channels, taps [C, taps], carried tails
};
constexpr int FEW_RPT = 16;      // state rows per thread: dim <= 8 * 16
template <bool DELTA>
__global__ void __launch_bounds__(256) hy_few_memory_kernel(FewArgs f, HyRows r) {
    HY_PDL();
    const BlockArgs& p = f.p;
    __shared__ __align__(16) float qs[BM_FEW][128], ks[BM_FEW][128], vs[BM_FEW][128], part[8][128], po[2][8][128];
    __shared__ float gb[BM_FEW][2];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, seq = blockIdx.x, h = blockIdx.y, D = p.D, VD = p.VD;
    const long long row0 = r.seq_row0[seq]; const int len = r.seq_row0[seq + 1] - (int)row0, pos0 = r.seq_pos0[seq], slot = r.seq_state[seq];
    if (len > BM_FEW) return;                            // the block form takes this sequence
    const int qh = h / (p.H / p.QH), c4 = lane * 4; const bool ok = c4 < VD;
    float* st = p.state + (((long long)slot * p.H + h) * D) * VD;
    float4 S[FEW_RPT];
#pragma unroll
    for (int i = 0; i < FEW_RPT; ++i) {
        const int d = warp + 8 * i;
        S[i] = (pos0 > 0 && ok && d < D) ? *reinterpret_cast<const float4*>(st + (long long)d * VD + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int n = 2 * D + VD;
    for (int i = tid; i < len * n; i += 256) {
        const int t = i / n, c = i - t * n;
        float* dst = c < D ? &qs[t][c] : c < 2 * D ? &ks[t][c - D] : &vs[t][c - 2 * D];
        if (DELTA) {                                     // channel of the convolution: [q heads | k heads | v heads]
            const int ch = c < D ? qh * D + c : c < 2 * D ? p.QH * D + qh * D + (c - D) : 2 * p.QH * D + h * VD + (c - 2 * D);
            const bf* tail = f.tails + (long long)slot * (f.taps - 1) * f.C;
            float acc = 0.f;
            for (int j = 0; j < f.taps; ++j) {
                const int src = t - (f.taps - 1) + j;
                const float x = src >= 0 ? ldf(f.in + (row0 + src) * p.ld_in + ch) : pos0 > 0 ? ldf(tail + (long long)(f.taps - 1 + src) * f.C + ch) : 0.f;
                acc = fmaf(f.conv_w[ch * f.taps + j], x, acc);
            }
            *dst = __bfloat162float(__float2bfloat16_rn(silu_fast_f32(acc)));      // as the convolution kernel leaves it
        } else *dst = c < D ? ldf(p.q + (row0 + t) * p.ld + (long long)h * D + c) : c < 2 * D ? ldf(p.k + (row0 + t) * p.ld + (long long)h * D + (c - D)) : ldf(p.v + (row0 + t) * p.ld + (long long)h * VD + (c - 2 * D));
    }
    if (tid < len) {
        if (DELTA) {
            const long long at = (row0 + tid) * p.ld_in + h;
            gb[tid][0] = expf(log_decay(p.A_log[h], ldf(p.a + at) + p.dt_bias[h])); gb[tid][1] = sigmoidf_(ldf(p.b + at));
        } else gb[tid][0] = p.decay[h];
    }
    __syncthreads();
    if (DELTA) {
        for (int u = warp; u < 2 * len; u += 8) {        // unit vectors
            float* x = u & 1 ? ks[u >> 1] : qs[u >> 1];
            float ss = 0.f;
            for (int c = lane; c < D; c += 32) ss = fmaf(x[c], x[c], ss);
            const float s = (u & 1 ? 1.0f : rsqrtf((float)D)) / sqrtf(warp_sum(ss) + 1e-6f);
            for (int c = lane; c < D; c += 32) x[c] *= s;
        }
        __syncthreads();
    }
    for (int t = 0; t < len; ++t) {
        const float g = gb[t][0];
        float4 u = ok ? *reinterpret_cast<const float4*>(&vs[t][c4]) : make_float4(0.f, 0.f, 0.f, 0.f), o = make_float4(0.f, 0.f, 0.f, 0.f);
        if (DELTA) {
            float4 dot = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < FEW_RPT; ++i) {
                const int d = warp + 8 * i;
                if (d < D) {
                    const float k = ks[t][d];
                    S[i].x *= g; S[i].y *= g; S[i].z *= g; S[i].w *= g;
                    dot.x = fmaf(S[i].x, k, dot.x); dot.y = fmaf(S[i].y, k, dot.y); dot.z = fmaf(S[i].z, k, dot.z); dot.w = fmaf(S[i].w, k, dot.w);
                }
            }
            *reinterpret_cast<float4*>(&part[warp][c4]) = dot;
            __syncthreads();
            dot = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int w = 0; w < 8; ++w) { const float4 x = *reinterpret_cast<const float4*>(&part[w][c4]); dot.x += x.x; dot.y += x.y; dot.z += x.z; dot.w += x.w; }
            const float be = gb[t][1];
            u = make_float4(be * (u.x - dot.x), be * (u.y - dot.y), be * (u.z - dot.z), be * (u.w - dot.w));
        }
#pragma unroll
        for (int i = 0; i < FEW_RPT; ++i) {
            const int d = warp + 8 * i;
            if (d < D) {
                const float k = ks[t][d], q = qs[t][d];
                if (!DELTA) { S[i].x *= g; S[i].y *= g; S[i].z *= g; S[i].w *= g; }
                S[i].x = fmaf(k, u.x, S[i].x); S[i].y = fmaf(k, u.y, S[i].y); S[i].z = fmaf(k, u.z, S[i].z); S[i].w = fmaf(k, u.w, S[i].w);
                o.x = fmaf(S[i].x, q, o.x); o.y = fmaf(S[i].y, q, o.y); o.z = fmaf(S[i].z, q, o.z); o.w = fmaf(S[i].w, q, o.w);
            }
        }
        *reinterpret_cast<float4*>(&po[t & 1][warp][c4]) = o;
        __syncthreads();
        if (warp == (t & 7)) {                           // one warp joins the token's read-out; its buffer is written again two tokens later, behind the next token's barrier
            o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int w = 0; w < 8; ++w) { const float4 x = *reinterpret_cast<const float4*>(&po[t & 1][w][c4]); o.x += x.x; o.y += x.y; o.z += x.z; o.w += x.w; }
            if (DELTA) {
                const float ss = warp_sum(ok ? (o.x * o.x + o.y * o.y) + (o.z * o.z + o.w * o.w) : 0.f), rr = 1.0f / sqrtf(ss / (float)VD + p.eps);
                if (ok) {
                    const uint2 gr = *reinterpret_cast<const uint2*>(p.gate + (row0 + t) * p.ld_in + (long long)h * VD + c4); const float4 w = *reinterpret_cast<const float4*>(p.norm_w + c4);
                    *reinterpret_cast<uint2*>(reinterpret_cast<bf*>(p.out) + (row0 + t) * p.ldo + (long long)h * VD + c4) =
                        make_uint2(pack_bf16x2(o.x * rr * w.x * siluf_(bf16lo(gr.x)), o.y * rr * w.y * siluf_(bf16hi(gr.x))), pack_bf16x2(o.z * rr * w.z * siluf_(bf16lo(gr.y)), o.w * rr * w.w * siluf_(bf16hi(gr.y))));
                }
            } else if (ok) *reinterpret_cast<float4*>(reinterpret_cast<float*>(p.out) + (row0 + t) * p.ldo + (long long)h * VD + c4) = o;
        }
    }
    if (ok)
#pragma unroll
        for (int i = 0; i < FEW_RPT; ++i) { const int d = warp + 8 * i; if (d < D) *reinterpret_cast<float4*>(st + (long long)d * VD + c4) = S[i]; }
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <bool DELTA>
cudaError_t block_launch(const BlockArgs& p, const HyRows& r, cudaStream_t s) {
    const int VP = (p.VD + 15) / 16 * 16, DP = p.D <= 64 ? 64 : 128;
    const BlockSmem L(DELTA, DP, VP);
    static bool done[4][16] = {};
    auto go = [&](auto kern, bool (&flag)[16], int threads) -> cudaError_t {
        if (cudaError_t e = ensure_dynamic_smem(kern, 160 * 1024, flag); e != cudaSuccess) return e;
        return launch_plain(kern, dim3(r.S, p.H), dim3(threads), (size_t)L.total, s, p, r);
    };
    if (VP <= 64) return DP == 64 ? go(hy_block_memory_kernel<DELTA, 64, 128>, done[0], 128) : go(hy_block_memory_kernel<DELTA, 128, 128>, done[1], 128);
    return DP == 64 ? go(hy_block_memory_kernel<DELTA, 64, 256>, done[2], 256) : go(hy_block_memory_kernel<DELTA, 128, 256>, done[3], 256);
}

}  // namespace

bool hy_block_memory_supported(int dim, int vdim) { return dim % 8 == 0 && vdim % 8 == 0 && dim >= 8 && vdim >= 8 && dim <= 128 && vdim <= 128; }

cudaError_t hy_lightning_mix(const HyBlockHead& m, const void* q, const void* k, const void* v, int ld, const float* decay, float* state, float* out, bool few, bool many, const HyRows& r,
                             cudaStream_t s) {
    if (r.T <= 0) return cudaSuccess;
    if (!hy_block_memory_supported(m.dim, m.vdim) || m.qk_heads != m.heads || ld % 8 || !al16(q) || !al16(k) || !al16(v) || !al16(state) || !al16(out)) return cudaErrorInvalidValue;
    BlockArgs p{}; p.q = (const bf*)q; p.k = (const bf*)k; p.v = (const bf*)v; p.ld = ld; p.decay = decay; p.state = state; p.out = out; p.ldo = m.heads * m.vdim;
    p.H = p.QH = m.heads; p.D = m.dim; p.VD = m.vdim;
    if (few) { FewArgs f{}; f.p = p; if (cudaError_t e = launch_plain(hy_few_memory_kernel<false>, dim3(r.S, m.heads), dim3(256), 0, s, f, r); e != cudaSuccess) return e; }
    return many ? block_launch<false>(p, r, s) : cudaSuccess;
}

cudaError_t hy_delta_mix(const HyBlockHead& m, const HyDeltaMix& d, float* state, void* out, int ldo, bool few, bool many, const HyRows& r, cudaStream_t s) {
    if (r.T <= 0) return cudaSuccess;
    if (!hy_block_memory_supported(m.dim, m.vdim) || m.qk_heads <= 0 || m.heads % m.qk_heads || d.ld_conv % 8 || d.ld_in % 8 || ldo % 8 || !al16(d.conv) || !al16(d.in) || !al16(d.gate) ||
        !al16(d.norm_w) || !al16(state) || !al16(out)) return cudaErrorInvalidValue;
    BlockArgs p{}; const int qk = m.qk_heads * m.dim;
    p.q = (const bf*)d.conv; p.k = p.q + qk; p.v = p.k + qk; p.ld = d.ld_conv; p.gate = (const bf*)d.gate; p.a = (const bf*)d.a; p.b = (const bf*)d.b; p.ld_in = d.ld_in;
    p.A_log = d.A_log; p.dt_bias = d.dt_bias; p.norm_w = d.norm_w; p.eps = d.eps; p.state = state; p.out = out; p.ldo = ldo; p.H = m.heads; p.QH = m.qk_heads; p.D = m.dim; p.VD = m.vdim;
    if (few) {
        FewArgs f{}; f.p = p; f.in = (const bf*)d.in; f.conv_w = d.conv_w; f.taps = d.taps; f.C = 2 * qk + m.heads * m.vdim; f.tails = (const bf*)d.tails;
        if (cudaError_t e = launch_plain(hy_few_memory_kernel<true>, dim3(r.S, m.heads), dim3(256), 0, s, f, r); e != cudaSuccess) return e;
    }
    return many ? block_launch<true>(p, r, s) : cudaSuccess;
}

}  // namespace oa
