// seq_mlstm.cu -- the matrix memory of xLSTM (mLSTM) for the token-major models: a linear-attention state with one input gate
// and one forget gate per head and token, both exponential, kept in range by a running maximum of their logarithms.  float32
// throughout (sums of log gates in double).  Per head, with keys of size D and values of size Dv:
//
//   i_t = c tanh((zi_t + bi) / c),  f_t = log sigmoid(c tanh((zf_t + bf) / c)),  m_t = max(f_t + m_(t-1), i_t)
//   S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T,   n_t the same with k_t alone
//   o_t = S_t^T q_t / (max(|n_t.q_t|, e^(-m_t)) + 1e-6);  then o / rms(o) * w * sigmoid(g)
//
// S [D][Dv], n [D] and m of every sequence slot are rows of the cache manager's state arrays.  A sequence whose first position is
// 0 starts from zero (m too), whatever its slot held.
//
//   step       one token per sequence: everything above in ONE launch.  A cluster of up to eight blocks owns a (sequence, head), a
//              block a slice of value columns; every block forms n.q itself, the root mean square meets over distributed shared
//              memory, and block 0 writes n and m once all blocks have read them.
//   prompts    chunks of 64 tokens, all at once.  With F the running sum of f inside a chunk,
//              m_t = max(F_t + m_in, max_(s<=t) (F_t - F_s + i_s)) for every t, so that
//              1. gates:   F, i, m of every token (a block per sequence and head: one scan of (sum, maximum) pairs);
//              2. update:  U_c = sum_s e^(F_end - F_s + i_s - m_end) k_s v_s^T per chunk (and the n part);
//              3. scan:    per state element over the chunks in order, leaving the state BEFORE each chunk in the workspace;
//              4. output:  o_t = e^(F_t + m_in - m_t) S_c^T q_t + sum_(s<=t) e^(F_t - F_s + i_s - m_t) (q_t.k_s) v_s over the
//                 denominator of the same form; with the head's values in one block the norm, weight and gate too.
//              A launch covers a segment of chunks (the host bounds the workspace); the state travels through the slot's rows.
#include <cooperative_groups.h>
#include "common.cuh"
#include "../../include/pgk_b200.h"

using namespace pgk;
namespace cg = cooperative_groups;

namespace {

struct MlstmArgs {
    const float* proj; int ld, q_off, k_off, v_off, g_off, i_off, f_off;
    const float* ib; const float* fb; float cap, q_scale;
    const float* w; float eps;           // [H * Dv] output weight
    float* out; int ldo;
    float* S; float* N; float* M;        // [slots][H][D][Dv], [slots][H][D], [slots][H]
    const int4* seqs;                    // (first row, rows, slot, first position)
    int H, D, Dv;
    int vec;                             // rows, offsets and sizes are multiples of 16 bytes
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float log_in(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget(float z, float cap) {
    const float c = cap * tanhf(z / cap);
    return fminf(c, 0.f) - log1pf(expf(-fabsf(c)));
}

// ---------------------------------------------------------------- one token per sequence
constexpr int ST = 256;                 // threads per block
constexpr int SROWS = 8;                // state rows in flight per thread

// VW value columns per thread and state row: 4 (16-byte rows) or 1
template <int VW>
__global__ void __launch_bounds__(ST) mlstm_step_kernel(MlstmArgs a, int slice) {
    extern __shared__ __align__(16) float sm[];
    const int D = a.D, Dv = a.Dv, D4 = (D + 3) & ~3;
    float* qs = sm;                      // [D4]
    float* ks = qs + D4;                 // [D4]
    float* red = ks + D4;                // [ST * VW]
    float* os = red + ST * VW;           // [slice]
    __shared__ float wred[ST / 32];
    __shared__ float part[2];            // this block's sum of squares
    cg::cluster_group cluster = cg::this_cluster();
    const int rank = (int)cluster.block_rank(), nb = (int)cluster.num_blocks();
    const int4 sq = a.seqs[blockIdx.x];
    const int slot = sq.z, h = blockIdx.y, c0 = rank * slice, nc = max(0, min(slice, Dv - c0));
    const bool fresh = sq.w == 0;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const float* row = a.proj + (size_t)sq.x * a.ld;
    const float* Nrow = a.N + ((size_t)slot * a.H + h) * D;
    const float m_old = fresh ? 0.f : a.M[(size_t)slot * a.H + h];
    const float zi = row[a.i_off + h] + a.ib[h], zf = row[a.f_off + h] + a.fb[h];

    // the thread's first state rows travel while the gates are formed
    const int CG = nc / VW, CGt = CG < ST ? CG : ST, RG = CGt > 0 ? ST / CGt : 1;
    const int cgi = CGt > 0 ? tid % CGt : 0, rg = CGt > 0 ? tid / CGt : 0;
    const bool act = CGt > 0 && rg < RG;
    float* Sg = a.S + ((size_t)slot * a.H + h) * D * Dv + c0;
    float pre[SROWS][VW];
    auto fetch = [&](float (&r)[SROWS][VW], int d0, int col) {
#pragma unroll
        for (int j = 0; j < SROWS; ++j) {
            const int d = d0 + j * RG;
            if (act && d < D && !fresh) {
                const float* p = Sg + (size_t)d * Dv + col;
                if (VW == 4) *(float4*)&r[j][0] = *(const float4*)p;
                else r[j][0] = *p;
            } else {
#pragma unroll
                for (int e = 0; e < VW; ++e) r[j][e] = 0.f;
            }
        }
    };
    fetch(pre, rg, cgi * VW);

    const float li = log_in(zi, a.cap), lf = log_forget(zf, a.cap);
    const float m = fmaxf(lf + m_old, li), fa = expf(lf + m_old - m), fb = expf(li - m);
    float nq = 0.f;
    for (int d = tid; d < D; d += ST) {
        const float q = row[a.q_off + (size_t)h * D + d] * a.q_scale, k = row[a.k_off + (size_t)h * D + d];
        qs[d] = q; ks[d] = k;
        const float n = fmaf(fa, fresh ? 0.f : Nrow[d], fb * k);
        nq = fmaf(n, q, nq);
    }
    nq = warp_sum(nq);
    if (lane == 0) wred[warp] = nq;
    __syncthreads();
    nq = 0.f;
#pragma unroll
    for (int i = 0; i < ST / 32; ++i) nq += wred[i];
    const float den = fmaxf(fabsf(nq), expf(-m)) + 1e-6f;

    float ss = 0.f;
    for (int cb = 0; cb < CG; cb += CGt) {                 // more column groups than threads: walk them
        const int col = (cb + cgi) * VW;
        const bool live = act && cb + cgi < CG;
        float v[VW], o[VW];
#pragma unroll
        for (int e = 0; e < VW; ++e) { v[e] = live ? fb * row[a.v_off + (size_t)h * Dv + c0 + col + e] : 0.f; o[e] = 0.f; }
        if (cb > 0) fetch(pre, rg, live ? col : 0);
        for (int d0 = rg; d0 < D; d0 += RG * SROWS) {
            float cur[SROWS][VW];
#pragma unroll
            for (int j = 0; j < SROWS; ++j)
#pragma unroll
                for (int e = 0; e < VW; ++e) cur[j][e] = pre[j][e];
            if (d0 + RG * SROWS < D) fetch(pre, d0 + RG * SROWS, live ? col : 0);
#pragma unroll
            for (int j = 0; j < SROWS; ++j) {
                const int d = d0 + j * RG;
                if (!live || d >= D) continue;
                const float k = ks[d], q = qs[d];
                float s[VW];
#pragma unroll
                for (int e = 0; e < VW; ++e) {
                    s[e] = fmaf(fa, cur[j][e], k * v[e]);
                    o[e] = fmaf(q, s[e], o[e]);
                }
                float* p = Sg + (size_t)d * Dv + col;
                if (VW == 4) *(float4*)p = make_float4(s[0], s[VW / 4], s[VW / 2], s[VW - 1]);
                else *p = s[0];
            }
        }
        __syncthreads();                                   // `red` is free again
        if (live) {
#pragma unroll
            for (int e = 0; e < VW; ++e) red[(rg * CGt + cgi) * VW + e] = o[e];
        }
        __syncthreads();
        const int ncols = min(CGt, CG - cb) * VW;
        for (int c = tid; c < ncols; c += ST) {
            float t = 0.f;
            for (int r = 0; r < RG; ++r) t += red[r * CGt * VW + c];
            t /= den;
            os[cb * VW + c] = t;
            ss = fmaf(t, t, ss);
        }
    }
    ss = warp_sum(ss);
    __syncthreads();
    if (lane == 0) wred[warp] = ss;
    __syncthreads();
    if (tid == 0) {
        float t = 0.f;
        for (int i = 0; i < ST / 32; ++i) t += wred[i];
        part[0] = t;
    }
    cluster.sync();                                        // every block has read n and m, and left its sum of squares
    float tot = 0.f;
    for (int b = 0; b < nb; ++b) tot += *cluster.map_shared_rank(&part[0], b);
    cluster.barrier_arrive();                              // a block's shared memory stays until all have read it
    if (rank == 0) {
        float* Nw = a.N + ((size_t)slot * a.H + h) * D;
        for (int d = tid; d < D; d += ST) Nw[d] = fmaf(fa, fresh ? 0.f : Nw[d], fb * ks[d]);
        if (tid == 0) a.M[(size_t)slot * a.H + h] = m;
    }
    const float inv = 1.f / sqrtf(tot / (float)Dv + a.eps);
    for (int c = tid; c < nc; c += ST) {
        const int hc = h * Dv + c0 + c;
        a.out[(size_t)sq.x * a.ldo + hc] = os[c] * inv * a.w[hc] * sigmoid_f(row[a.g_off + hc]);
    }
    cluster.barrier_wait();
}

// ---------------------------------------------------------------- prompts: gates
constexpr int MC = 64;                   // tokens per chunk
constexpr int MP = MC + 4;               // row stride of transposed tiles [dim][MC]

struct GateWs {                          // per (row, head), row-major [T][H]
    double* F;                           // sum of f from the chunk's first token to this one
    float* gi; float* m; float* mp;      // i, m, and m before the token
};

constexpr int GT = 256;                  // tokens per round of the gate scan, one per thread

// A block per (sequence, head): every round takes GT tokens, scans (sum of f, running maximum) pairs inside the warps, then over the
// warps' totals.  (F1, m1) then (F2, m2) compose to (F1 + F2, max(m1 + F2, m2)).
__global__ void __launch_bounds__(GT) mlstm_gates_kernel(MlstmArgs a, GateWs g) {
    __shared__ double wF[GT / 32], wm[GT / 32], Fat[GT / MC], last_m;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y;
    const int4 sq = a.seqs[blockIdx.x];
    float* Mrow = a.M + (size_t)sq.z * a.H + h;
    double m_in = sq.w > 0 ? (double)*Mrow : 0.0;
    const float ib = a.ib[h], fb = a.fb[h];
    float zi = 0.f, zf = 0.f;
    if (tid < sq.y) {
        const float* row = a.proj + (size_t)(sq.x + tid) * a.ld;
        zi = row[a.i_off + h]; zf = row[a.f_off + h];
    }
    for (int t0 = 0; t0 < sq.y; t0 += GT) {
        const int t = t0 + tid;
        const bool in = t < sq.y;
        const float li = log_in(zi + ib, a.cap), lf = log_forget(zf + fb, a.cap);
        if (t + GT < sq.y) {                               // the next round's logits travel meanwhile
            const float* row = a.proj + (size_t)(sq.x + t + GT) * a.ld;
            zi = row[a.i_off + h]; zf = row[a.f_off + h];
        }
        double F = in ? (double)lf : 0.0, mx = in ? (double)li : -1e300;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double Fp = __shfl_up_sync(0xffffffffu, F, o), mxp = __shfl_up_sync(0xffffffffu, mx, o);
            if (lane >= o) { mx = fmax(mx, mxp + F); F += Fp; }
        }
        __syncthreads();                                   // the round before has read the shared arrays
        if (lane == 31) { wF[warp] = F; wm[warp] = mx; }
        __syncthreads();
        double Fw = 0.0, mw = m_in;                        // F and m before this warp's tokens
        for (int w = 0; w < warp; ++w) { mw = fmax(mw + wF[w], wm[w]); Fw += wF[w]; }
        const double m = fmax(F + mw, mx);
        double mp = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) mp = mw;
        if (tid % MC == 0) Fat[tid / MC] = Fw;             // the sum in front of every chunk of the round
        if (t == min(sq.y, t0 + GT) - 1) last_m = m;
        __syncthreads();
        if (in) {
            const size_t at = (size_t)(sq.x + t) * a.H + h;
            g.F[at] = Fw - Fat[tid / MC] + F; g.gi[at] = li; g.m[at] = (float)m; g.mp[at] = (float)mp;
        }
        m_in = last_m;
    }
    if (tid == 0) *Mrow = (float)m_in;
}

// ---------------------------------------------------------------- prompts: chunk update
struct ChunkArgs {
    MlstmArgs a; GateWs g;
    float* ws;                           // [sequences][grid.x chunks][H][D * Dv + D]
    int c_begin, chunks, slices, fuse;   // slices of value columns per head (at most SLICE_MAX each)
};
constexpr int SLICE_MAX = 128;

__host__ __device__ __forceinline__ int round4(int n) { return (n + 3) & ~3; }
__device__ __forceinline__ size_t chunk_row(const ChunkArgs& c, int seq, int chunk, int h) {
    return (((size_t)seq * c.chunks + chunk) * c.a.H + h) * ((size_t)c.a.D * c.a.Dv + c.a.D);
}

// rows r0 .. r0 + MC - 1 (zeros from nc on) of `cols` columns at `src` into shared memory, row stride ls
__device__ __forceinline__ void stage_rows(const float* src, int ld, int nc, int cols, float* dst, int ls, bool vec) {
    if (vec) {
        const int c4 = ls >> 2;
        for (int i = threadIdx.x; i < MC * c4; i += 256) {
            const int r = i / c4, c = (i - r * c4) * 4;
            if (r < nc && c < cols) cp_async16(dst + r * ls + c, src + (size_t)r * ld + c);
            else *(float4*)(dst + r * ls + c) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
        for (int i = threadIdx.x; i < MC * ls; i += 256) {
            const int r = i / ls, c = i - r * ls;
            dst[i] = (r < nc && c < cols) ? src[(size_t)r * ld + c] : 0.f;
        }
    }
}

__global__ void __launch_bounds__(256, 2) mlstm_update_kernel(ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    const MlstmArgs& a = p.a;
    const int D = a.D, Dv = a.Dv, D8 = (D + 7) & ~7;
    const int h = blockIdx.z / p.slices, sl = blockIdx.z - h * p.slices;
    const int cw = (round4(Dv) / 4 + p.slices - 1) / p.slices * 4, v0 = sl * cw, nv = min(cw, Dv - v0);
    float* Ks = sm;                      // [MC][D8]
    float* Vs = Ks + MC * D8;            // [MC][cw], rows scaled by their weight
    __shared__ float us[MC];
    const int4 sq = a.seqs[blockIdx.y];
    const int c = p.c_begin + blockIdx.x, tid = threadIdx.x;
    if (c * MC >= sq.y || nv <= 0) return;
    const int nc = min(MC, sq.y - c * MC), r0 = sq.x + c * MC;
    stage_rows(a.proj + (size_t)r0 * a.ld + a.k_off + (size_t)h * D, a.ld, nc, D, Ks, D8, a.vec);
    stage_rows(a.proj + (size_t)r0 * a.ld + a.v_off + (size_t)h * Dv + v0, a.ld, nc, nv, Vs, cw, a.vec);
    cp_async_commit();
    if (tid < MC) {
        float u = 0.f;
        if (tid < nc) {
            const size_t at = (size_t)(r0 + tid) * a.H + h, ae = (size_t)(r0 + nc - 1) * a.H + h;
            u = expf((float)(p.g.F[ae] - p.g.F[at] + (double)p.g.gi[at] - (double)p.g.m[ae]));
        }
        us[tid] = u;
    }
    cp_async_wait<0>();
    __syncthreads();
    for (int i = tid; i < MC * cw; i += 256) Vs[i] *= us[i / cw];
    __syncthreads();
    float* U = p.ws + chunk_row(p, blockIdx.y, blockIdx.x, h);
    const int nTv = cw / 4, ntiles = (D8 / 8) * nTv;
    const bool st4 = a.vec && (D & 3) == 0;
    for (int tile = tid; tile < ntiles; tile += 256) {
        const int d0 = (tile / nTv) * 8, w0 = (tile % nTv) * 4;
        float acc[8][4] = {};
#pragma unroll 2
        for (int s = 0; s < nc; ++s) {
            const float4 ka = *(const float4*)(Ks + s * D8 + d0), kb = *(const float4*)(Ks + s * D8 + d0 + 4);
            const float4 v4 = *(const float4*)(Vs + s * cw + w0);
            const float kk[8] = {ka.x, ka.y, ka.z, ka.w, kb.x, kb.y, kb.z, kb.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(kk[i], vv[j], acc[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (d0 + i >= D) break;
            float* dst = U + (size_t)(d0 + i) * Dv + v0 + w0;
            if (st4 && w0 + 3 < nv) *(float4*)dst = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
            else
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (w0 + j < nv) dst[j] = acc[i][j];
        }
    }
    if (sl == 0)
        for (int d = tid; d < D; d += 256) {
            float n = 0.f;
            for (int s = 0; s < nc; ++s) n = fmaf(us[s], Ks[s * D8 + d], n);
            U[(size_t)D * Dv + d] = n;
        }
}

// ---------------------------------------------------------------- prompts: scan over the chunks, one thread per state element
__global__ void __launch_bounds__(256) mlstm_scan_kernel(ChunkArgs p) {
    const MlstmArgs& a = p.a;
    __shared__ float dec[256];
    const size_t mat = (size_t)a.D * a.Dv, per = mat + a.D, e = (size_t)blockIdx.x * 256 + threadIdx.x;
    const int h = blockIdx.y;
    const int4 sq = a.seqs[blockIdx.z];
    const int nchunks = (sq.y + MC - 1) / MC, cend = min(nchunks, p.c_begin + p.chunks);
    if (p.c_begin >= nchunks) return;
    const bool live = e < per;
    float* St = e < mat ? a.S + ((size_t)sq.z * a.H + h) * mat + e : a.N + ((size_t)sq.z * a.H + h) * a.D + (e - mat);
    float S = (live && (sq.w > 0 || p.c_begin > 0)) ? *St : 0.f;
    float* u0 = p.ws + chunk_row(p, blockIdx.z, 0, h) + e;
    const size_t step = (size_t)a.H * per;
    constexpr int B = 8;                                   // loads in flight per thread
    for (int cb = p.c_begin; cb < cend; cb += 256) {
        const int nb = min(256, cend - cb);
        __syncthreads();
        if ((int)threadIdx.x < nb) {                       // the chunks' decays e^(F_end + m_in - m_end)
            const int c = cb + threadIdx.x, r0 = sq.x + c * MC, re = sq.x + min(sq.y, (c + 1) * MC) - 1;
            const size_t as = (size_t)r0 * a.H + h, ae = (size_t)re * a.H + h;
            dec[threadIdx.x] = expf((float)(p.g.F[ae] + (double)p.g.mp[as] - (double)p.g.m[ae]));
        }
        __syncthreads();
        if (!live) continue;
        for (int c = 0; c < nb; c += B) {
            float add[B];
            float* u = u0 + (size_t)(cb - p.c_begin + c) * step;
#pragma unroll
            for (int i = 0; i < B; ++i) add[i] = c + i < nb ? __ldcg(u + (size_t)i * step) : 0.f;
#pragma unroll
            for (int i = 0; i < B; ++i)
                if (c + i < nb) {
                    __stcg(u + (size_t)i * step, S);
                    S = fmaf(S, dec[c + i], add[i]);
                }
        }
    }
    if (live) *St = S;
}

// ---------------------------------------------------------------- prompts: outputs of a chunk
constexpr int SLAB = 16;                 // state rows per slab

// q or k rows transposed into [D][MP]: a warp moves 8 consecutive elements of 4 rows at a time (whole sectors, no bank conflicts)
__device__ __forceinline__ void stage_transposed(const float* src, int ld, int nc, int D, float mult, float* dst) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, dl = lane & 7, tl = lane >> 3;
    const int nd = (D + 7) / 8;
    constexpr int B = 8;                                   // loads in flight per thread
    for (int u0 = warp; u0 < nd * (MC / 4); u0 += 8 * B) {
        float r[B];
#pragma unroll
        for (int b = 0; b < B; ++b) {
            const int u = u0 + 8 * b, d = (u % nd) * 8 + dl, t = (u / nd) * 4 + tl;
            r[b] = (d < D && t < nc) ? __ldg(src + (size_t)t * ld + d) : 0.f;
        }
#pragma unroll
        for (int b = 0; b < B; ++b) {
            const int u = u0 + 8 * b, d = (u % nd) * 8 + dl, t = (u / nd) * 4 + tl;
            if (d < D && t < MC) dst[d * MP + t] = r[b] * mult;
        }
    }
}

__global__ void __launch_bounds__(256, 2) mlstm_output_kernel(ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    const MlstmArgs& a = p.a;
    const int D = a.D, Dv = a.Dv;
    const int h = blockIdx.z / p.slices, sl = blockIdx.z - h * p.slices;
    const int cw = (round4(Dv) / 4 + p.slices - 1) / p.slices * 4, v0 = sl * cw, nv = min(cw, Dv - v0);
    const int r1 = max(D * MP, MC * cw);
    float* Qt = sm;                      // [D][MP]
    float* R1 = Qt + D * MP;             // K transposed [D][MP], then V [MC][cw], then the outputs [MC][cw]
    float* At = R1 + r1;                 // [MC][MP]: weight of key s for query t at [s][t]
    float* slab = At + MC * MP;          // [2][SLAB][cw]
    // the exponent F_t - F_s + i_s - m_t = (F_t - m_t) + (i_s - F_s), either part as a pair of floats: the sum of the leading parts
    // is rounded relative to the exponent itself, however large F has grown
    __shared__ float2 rt[MC], cs[MC];
    __shared__ float ms[MC], win[MC], den[MC];
    const int4 sq = a.seqs[blockIdx.y];
    const int c = p.c_begin + blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (c * MC >= sq.y || nv <= 0) return;
    const int nc = min(MC, sq.y - c * MC), r0 = sq.x + c * MC;
    const bool has_state = sq.w > 0 || c > 0;
    const float* Sc = p.ws + chunk_row(p, blockIdx.y, blockIdx.x, h);
    const bool sv = a.vec && (D & 3) == 0;
    auto fetch_slab = [&](int b) {                         // slab b of the starting state
        float* dst = slab + (b & 1) * SLAB * cw;
        const int d0 = b * SLAB, rows = min(SLAB, D - d0);
        if (sv) {
            const int c4 = cw >> 2;
            for (int i = tid; i < SLAB * c4; i += 256) {
                const int r = i / c4, cc = (i - r * c4) * 4;
                if (r < rows && cc < nv) cp_async16(dst + r * cw + cc, Sc + (size_t)(d0 + r) * Dv + v0 + cc);
                else *(float4*)(dst + r * cw + cc) = make_float4(0.f, 0.f, 0.f, 0.f);
            }
        } else {
            for (int i = tid; i < SLAB * cw; i += 256) {
                const int r = i / cw, cc = i - r * cw;
                if (r < rows && cc < nv) cp_async4(dst + i, Sc + (size_t)(d0 + r) * Dv + v0 + cc);
                else dst[i] = 0.f;
            }
        }
        cp_async_commit();
    };
    if (has_state) fetch_slab(0);
    const float* rows = a.proj + (size_t)r0 * a.ld;
    stage_transposed(rows + a.q_off + (size_t)h * D, a.ld, nc, D, a.q_scale, Qt);
    stage_transposed(rows + a.k_off + (size_t)h * D, a.ld, nc, D, 1.f, R1);
    if (tid < MC) {
        const size_t at = (size_t)(r0 + min(tid, nc - 1)) * a.H + h;
        const double F = p.g.F[at];
        const float m = p.g.m[at];
        const double r = F - (double)m, c0 = (double)p.g.gi[at] - F;
        rt[tid] = make_float2((float)r, (float)(r - (double)(float)r));
        cs[tid] = make_float2((float)c0, (float)(c0 - (double)(float)c0));
        ms[tid] = m;
        win[tid] = has_state ? expf((float)(F + (double)p.g.mp[(size_t)r0 * a.H + h] - (double)m)) : 0.f;
    }
    __syncthreads();
    {   // weights inside the chunk: 4 queries x 4 keys per thread
        const int t0 = (tid >> 4) * 4, s0 = (tid & 15) * 4;
        float acc[4][4] = {};
        if (s0 <= t0) {
#pragma unroll 4
            for (int d = 0; d < D; ++d) {
                const float4 q4 = *(const float4*)(Qt + d * MP + t0), k4 = *(const float4*)(R1 + d * MP + s0);
                const float qq[4] = {q4.x, q4.y, q4.z, q4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(qq[i], kk[j], acc[i][j]);
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float2 r = rt[t0 + i], c2 = cs[s0 + j];
                    acc[i][j] = (s0 + j <= t0 + i && t0 + i < nc) ? acc[i][j] * expf((r.x + c2.x) + (r.y + c2.y)) : 0.f;
                }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float r[4] = {acc[0][j], acc[1][j], acc[2][j], acc[3][j]};
            *(float4*)(At + (s0 + j) * MP + t0) = make_float4(r[0], r[1], r[2], r[3]);
        }
    }
    __syncthreads();                                       // K is done: V takes its place
    stage_rows(rows + a.v_off + (size_t)h * Dv + v0, a.ld, nc, nv, R1, cw, a.vec);
    cp_async_commit();
    {   // denominators: four threads per query
        const int t = tid >> 2, q = tid & 3;
        const float* Nc = Sc + (size_t)D * Dv;
        float x = 0.f, y = 0.f;
#pragma unroll 4
        for (int s = q; s <= t; s += 4) x += At[s * MP + t];
        if (has_state)
#pragma unroll 8
            for (int d = q; d < D; d += 4) y = fmaf(Qt[d * MP + t], __ldg(Nc + d), y);
        x = fmaf(y, win[t], x);
        x += __shfl_xor_sync(0xffffffffu, x, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2);
        if (q == 0) den[t] = fmaxf(fabsf(x), expf(-ms[t])) + 1e-6f;
    }
    const int nTv = cw / 4;
    const bool live = tid < 8 * nTv;
    const int t0 = live ? (tid / nTv) * 8 : 0, w0 = live ? (tid % nTv) * 4 : 0;
    float acc[8][4] = {};
    if (has_state) {
        const int nslab = (D + SLAB - 1) / SLAB;
        for (int b = 0; b < nslab; ++b) {
            if (b + 1 < nslab) fetch_slab(b + 1);          // travels while this one is used
            if (b == 0) cp_async_wait<0>();                // V and the first slabs
            else if (b + 1 < nslab) cp_async_wait<1>();
            else cp_async_wait<0>();
            __syncthreads();
            if (live) {
                const float* sb = slab + (b & 1) * SLAB * cw + w0;
                const int nd = min(SLAB, D - b * SLAB);
#pragma unroll 4
                for (int d = 0; d < nd; ++d) {
                    const float* qr = Qt + (b * SLAB + d) * MP + t0;
                    const float4 qa = *(const float4*)qr, qb = *(const float4*)(qr + 4), s4 = *(const float4*)(sb + d * cw);
                    const float qq[8] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w}, ss[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
                    for (int i = 0; i < 8; ++i)
#pragma unroll
                        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(qq[i], ss[j], acc[i][j]);
                }
            }
            __syncthreads();
        }
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] *= win[t0 + i];
    } else {
        cp_async_wait<0>();
        __syncthreads();
    }
    if (live) {
        const int send = min(nc, t0 + 8);
#pragma unroll 2
        for (int s = 0; s < send; ++s) {
            const float* ar = At + s * MP + t0;
            const float4 aa = *(const float4*)ar, ab = *(const float4*)(ar + 4), v4 = *(const float4*)(R1 + s * cw + w0);
            const float ww[8] = {aa.x, aa.y, aa.z, aa.w, ab.x, ab.y, ab.z, ab.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ww[i], vv[j], acc[i][j]);
        }
    }
    __syncthreads();                                       // V is done: the outputs take its place
    if (live)
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float r = 1.f / den[t0 + i];
            *(float4*)(R1 + (t0 + i) * cw + w0) = make_float4(acc[i][0] * r, acc[i][1] * r, acc[i][2] * r, acc[i][3] * r);
        }
    __syncthreads();
    for (int t = warp; t < nc; t += 8) {                   // a warp per row: norm, weight, gate (or the plain output)
        const float* o = R1 + t * cw;
        float* dst = a.out + (size_t)(r0 + t) * a.ldo + (size_t)h * Dv + v0;
        if (!p.fuse) {
            for (int v = lane; v < nv; v += 32) dst[v] = o[v];
            continue;
        }
        float q = 0.f;
        for (int v = lane; v < nv; v += 32) q = fmaf(o[v], o[v], q);
        const float inv = 1.f / sqrtf(warp_sum(q) / (float)Dv + a.eps);
        const float* gr = a.proj + (size_t)(r0 + t) * a.ld + a.g_off + (size_t)h * Dv;
        for (int v = lane; v < nv; v += 32) dst[v] = o[v] * inv * a.w[h * Dv + v] * sigmoid_f(gr[v]);
    }
}

inline bool mult4(long long v) { return (v & 3) == 0; }
inline bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

template <int VW>
int launch_step(const MlstmArgs& a, int n_seqs, int blocks, int slice, cudaStream_t st) {
    const size_t smem = sizeof(float) * (2 * (size_t)round4(a.D) + (size_t)ST * VW + (size_t)slice + 4);
    PGK_REQUIRE(smem <= 200 * 1024, "seq_mlstm_step failed: heads of %d x %d need %zu bytes of shared memory", a.D, a.Dv, smem);
    static bool configured = false;
    if (smem > 40 * 1024 && !configured) {
        PGK_CUDA(cudaFuncSetAttribute(mlstm_step_kernel<VW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        configured = true;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(n_seqs, a.H, blocks);
    cfg.blockDim = dim3(ST);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = blocks;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    count_launch();
    PGK_CUDA(cudaLaunchKernelEx(&cfg, mlstm_step_kernel<VW>, a, slice));
    return 0;
}

}  // namespace

extern "C" {

int pgk_seq_mlstm_chunk_tokens(void) { return MC; }

int pgk_seq_mlstm_fused_finish(int vdim) { return vdim <= SLICE_MAX ? 1 : 0; }

size_t pgk_seq_mlstm_gate_floats(int tokens, int heads) { return (size_t)tokens * heads * 5; }

static int fill_args(MlstmArgs& a, const char* who, const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, int i_off,
                     int f_off, const float* i_bias, const float* f_bias, float cap, float q_scale, const float* weight, float eps,
                     float* out, int ldo, float* S, float* N, float* M, const int32_t* seqs, int heads, int dim, int vdim) {
    PGK_REQUIRE(heads > 0 && dim > 0 && vdim > 0 && cap > 0.f, "%s failed: %d heads of %d x %d, gate cap %g", who, heads, dim, vdim, (double)cap);
    PGK_REQUIRE(proj && i_bias && f_bias && weight && out && S && N && M && seqs, "%s failed: a missing operand", who);
    a = MlstmArgs{proj, ld, q_off, k_off, v_off, g_off, i_off, f_off, i_bias, f_bias, cap, q_scale, weight, eps, out, ldo, S, N, M,
                  (const int4*)seqs, heads, dim, vdim, 0};
    a.vec = mult4(ld) && mult4(k_off) && mult4(v_off) && mult4(dim) && mult4(vdim) && aligned16(proj) && aligned16(S);
    return 0;
}

int pgk_seq_mlstm_step(const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, int i_off, int f_off,
                       const float* i_bias, const float* f_bias, float cap, float q_scale, const float* weight, float eps, float* out,
                       int ldo, float* S, float* N, float* M, const int32_t* seqs, int n_seqs, int heads, int dim, int vdim,
                       void* stream) {
    MlstmArgs a;
    if (fill_args(a, "seq_mlstm_step", proj, ld, q_off, k_off, v_off, g_off, i_off, f_off, i_bias, f_bias, cap, q_scale, weight, eps,
                  out, ldo, S, N, M, seqs, heads, dim, vdim)) return 1;
    if (n_seqs <= 0) return 0;
    // value columns are cut over a cluster until the grid fills the GPU, never into slices of fewer than 16
    int blocks = 1;
    while (blocks < 8 && (long long)n_seqs * heads * blocks < 148 && vdim / (2 * blocks) >= 16) blocks *= 2;
    const int slice = ((vdim + blocks - 1) / blocks + 3) & ~3;
    return mult4(vdim) && aligned16(S) ? launch_step<4>(a, n_seqs, blocks, slice, (cudaStream_t)stream)
                                       : launch_step<1>(a, n_seqs, blocks, slice, (cudaStream_t)stream);
}

int pgk_seq_mlstm_gates(const float* proj, int ld, int i_off, int f_off, const float* i_bias, const float* f_bias, float cap,
                        float* M, const int32_t* seqs, int n_seqs, int tokens, int heads, float* gates, void* stream) {
    PGK_REQUIRE(heads > 0 && cap > 0.f && gates && ((uintptr_t)gates & 7) == 0, "seq_mlstm_gates failed: %d heads, gate cap %g", heads, (double)cap);
    if (n_seqs <= 0 || tokens <= 0) return 0;
    MlstmArgs a{};
    a.proj = proj; a.ld = ld; a.i_off = i_off; a.f_off = f_off; a.ib = i_bias; a.fb = f_bias; a.cap = cap; a.M = M;
    a.seqs = (const int4*)seqs; a.H = heads;
    const size_t n = (size_t)tokens * heads;
    GateWs g{(double*)gates, gates + 2 * n, gates + 3 * n, gates + 4 * n};
    PGK_CUDA(launch(mlstm_gates_kernel, dim3(n_seqs, heads), dim3(GT), 0, (cudaStream_t)stream, a, g));
    return 0;
}

int pgk_seq_mlstm_chunks(const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, int i_off, int f_off,
                         const float* i_bias, const float* f_bias, float cap, float q_scale, const float* weight, float eps, float* out,
                         int ldo, float* S, float* N, float* M, const int32_t* seqs, int n_seqs, int tokens, int heads, int dim, int vdim,
                         const float* gates, int chunk_begin, int chunks, float* workspace, void* stream) {
    ChunkArgs p{};
    if (fill_args(p.a, "seq_mlstm_chunks", proj, ld, q_off, k_off, v_off, g_off, i_off, f_off, i_bias, f_bias, cap, q_scale, weight, eps,
                  out, ldo, S, N, M, seqs, heads, dim, vdim)) return 1;
    PGK_REQUIRE(gates && workspace && chunk_begin >= 0, "seq_mlstm_chunks failed: a missing workspace");
    if (n_seqs <= 0 || chunks <= 0) return 0;
    const size_t n = (size_t)tokens * heads;
    float* gt = const_cast<float*>(gates);
    p.g = GateWs{(double*)gt, gt + 2 * n, gt + 3 * n, gt + 4 * n};
    p.a.vec = p.a.vec && aligned16(workspace);
    p.ws = workspace; p.c_begin = chunk_begin; p.chunks = chunks;
    p.slices = (vdim + SLICE_MAX - 1) / SLICE_MAX;
    p.fuse = p.slices == 1;
    const int cw = (round4(vdim) / 4 + p.slices - 1) / p.slices * 4, D8 = (dim + 7) & ~7;
    const size_t smem2 = sizeof(float) * ((size_t)MC * D8 + (size_t)MC * cw);
    const size_t r1 = (size_t)dim * MP > (size_t)MC * cw ? (size_t)dim * MP : (size_t)MC * cw;
    const size_t smem4 = sizeof(float) * ((size_t)dim * MP + r1 + (size_t)MC * MP + 2 * (size_t)SLAB * cw);
    PGK_REQUIRE(smem2 <= 224 * 1024 && smem4 <= 224 * 1024, "seq_mlstm_chunks failed: keys of %d need %zu bytes of shared memory", dim, smem4);
    static bool configured = false;
    if (!configured) {
        PGK_CUDA(cudaFuncSetAttribute(mlstm_update_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
        PGK_CUDA(cudaFuncSetAttribute(mlstm_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
        configured = true;
    }
    cudaStream_t st = (cudaStream_t)stream;
    const dim3 grid(chunks, n_seqs, heads * p.slices);
    PGK_CUDA(launch(mlstm_update_kernel, grid, dim3(256), smem2, st, p));
    const size_t per = (size_t)dim * vdim + dim;
    PGK_CUDA(launch(mlstm_scan_kernel, dim3((unsigned)((per + 255) / 256), heads, n_seqs), dim3(256), 0, st, p));
    PGK_CUDA(launch(mlstm_output_kernel, grid, dim3(256), smem4, st, p));
    return 0;
}

}  // extern "C"
