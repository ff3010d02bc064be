// seq_gla.cu -- gated linear attention for the token-major models: a linear-attention state whose decay is a number per head, token
// AND key channel, formed from the token through a product of low inner size.  float32 throughout.  Per head, with keys of size D
// and values of size Dv:
//
//   a_t = sigmoid(W2 y_t + b)^(1 / tau)          (y_t: the inner columns of the fused projection, W2 [r x H D])
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t;  then o / rms(o) * w * silu(g)
//
// S [D][Dv] of every sequence slot is a row of the cache manager's state array.  A sequence whose first position is 0 starts from
// zero, whatever its slot held.
//
//   step       one token per sequence: everything above in ONE launch.  A cluster of up to eight blocks owns a (sequence, head), a
//              block a slice of value columns; the root mean square meets over distributed shared memory.
//   prompts    chunks of MC tokens, all at once, each cut into sub-chunks of SUB.  With g = log2 a, L_t the sum of g from the start
//              of t's sub-chunk to t, and E_j the sum over all of sub-chunk j (one number per channel each):
//              1. decays:  L of every token (a thread per channel walks a sub-chunk);
//              2. update:  U_c = sum_s 2^(sum of g behind s) k_s v_s^T per chunk, and the chunk's decay 2^(E_0 + E_1 + ..);
//              3. scan:    per state element over the chunks in order, leaving the state BEFORE each chunk in the workspace;
//              4. output:  o_t = (q_t 2^(sum of g up to t))^T S_c + sum_(s<=t) A_ts v_s with A_ts = sum_d q_td k_sd 2^(sum of g in (s, t]).
//                 Inside a sub-chunk the exponent is L_t - L_s; between sub-chunks i > j it is L_t + (E between) + (E_j - L_s), three
//                 factors that are at most 1 each.  So no exponent is ever positive, however strong the decays, and every
//                 difference is taken between sums over at most SUB tokens.
//              A launch covers a segment of chunks (the host bounds the workspace); the state travels through the slot's rows.
#include <cooperative_groups.h>
#include "common.cuh"
#include "../../include/pgk_b200.h"

using namespace pgk;
namespace cg = cooperative_groups;

namespace {

struct GlaArgs {
    const float* proj; int ld, q_off, k_off, v_off, g_off, y_off;
    const float* w2; const float* b2; int r; float inv_tau, q_scale;     // w2 [r][H * D]
    const float* w; float eps;           // [H * Dv] output weight
    float* out; int ldo;
    float* S;                            // [slots][H][D][Dv]
    const int4* seqs;                    // (first row, rows, slot, first position)
    int H, D, Dv;
    int vec;                             // rows, offsets and sizes are multiples of 16 bytes
};

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
constexpr float LOG2E = 1.44269504088896340736f;
// 2^x for decays: numbers too small to be normal count as zero
__device__ __forceinline__ float exp2_f(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}

// ---------------------------------------------------------------- one token per sequence
constexpr int ST = 256;                 // threads per block
constexpr int SROWS = 8;                // state rows in flight per thread

// VW value columns per thread and state row: 4 (16-byte rows) or 1
template <int VW>
__global__ void __launch_bounds__(ST) gla_step_kernel(GlaArgs a, int slice) {
    extern __shared__ __align__(16) float sm[];
    const int D = a.D, Dv = a.Dv, D4 = (D + 3) & ~3;
    float* qs = sm;                      // [D4]
    float* ks = qs + D4;                 // [D4]
    float* as = ks + D4;                 // [D4] decays
    float* red = as + D4;                // [ST * VW]
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

    // the thread's first state rows travel while the decays are formed
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

    for (int d = tid; d < D; d += ST) {
        qs[d] = row[a.q_off + (size_t)h * D + d] * a.q_scale;
        ks[d] = row[a.k_off + (size_t)h * D + d];
    }
    // decays: enough threads per channel to keep the loads of W2 in flight side by side
    int parts = 1;
    while (parts < 8 && D * parts * 2 <= ST && parts * 2 <= a.r) parts *= 2;
    for (int i0 = 0; i0 < D * parts; i0 += ST) {
        const int i = i0 + tid, d = i / parts, p = i - d * parts;
        float z = 0.f;
        if (d < D) {
            const float* wp = a.w2 + (size_t)h * D + d;
            const size_t hd = (size_t)a.H * D;
#pragma unroll 8
            for (int j = p; j < a.r; j += parts) z = fmaf(__ldg(wp + (size_t)j * hd), row[a.y_off + j], z);
        }
        for (int o = 1; o < parts; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
        if (d < D && p == 0) as[d] = expf(log_sigmoid(z + a.b2[(size_t)h * D + d]) * a.inv_tau);
    }
    __syncthreads();

    float ss = 0.f;
    for (int cb = 0; cb < CG; cb += CGt) {                 // more column groups than threads: walk them
        const int col = (cb + cgi) * VW;
        const bool live = act && cb + cgi < CG;
        float v[VW], o[VW];
#pragma unroll
        for (int e = 0; e < VW; ++e) { v[e] = live ? row[a.v_off + (size_t)h * Dv + c0 + col + e] : 0.f; o[e] = 0.f; }
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
                const float k = ks[d], q = qs[d], dec = as[d];
                float s[VW];
#pragma unroll
                for (int e = 0; e < VW; ++e) {
                    s[e] = fmaf(dec, cur[j][e], k * v[e]);
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
    cluster.sync();                                        // every block has left its sum of squares
    float tot = 0.f;
    for (int b = 0; b < nb; ++b) tot += *cluster.map_shared_rank(&part[0], b);
    cluster.barrier_arrive();                              // a block's shared memory stays until all have read it
    const float inv = 1.f / sqrtf(tot / (float)Dv + a.eps);
    for (int c = tid; c < nc; c += ST) {
        const int hc = h * Dv + c0 + c;
        a.out[(size_t)sq.x * a.ldo + hc] = os[c] * inv * a.w[hc] * silu_f(row[a.g_off + hc]);
    }
    cluster.barrier_wait();
}

// ---------------------------------------------------------------- prompts: decays
constexpr int SUB = 16;                  // tokens per sub-chunk

// A thread per channel and sub-chunk: L[t][h D + d], the running sum of log2 a inside the sub-chunk
__global__ void __launch_bounds__(256) gla_decays_kernel(GlaArgs a, float* L) {
    extern __shared__ __align__(16) float ys[];            // [r][SUB]
    const int4 sq = a.seqs[blockIdx.z];
    const int t0 = blockIdx.x * SUB;
    if (t0 >= sq.y) return;
    const int n = min(SUB, sq.y - t0), r0 = sq.x + t0, hd = a.H * a.D;
    for (int i = threadIdx.x; i < a.r * SUB; i += 256) {
        const int t = i / a.r, j = i - t * a.r;
        ys[j * SUB + t] = t < n ? a.proj[(size_t)(r0 + t) * a.ld + a.y_off + j] : 0.f;
    }
    __syncthreads();
    const int c = blockIdx.y * 256 + threadIdx.x;
    if (c >= hd) return;
    float z[SUB];
    const float b = a.b2[c];
#pragma unroll
    for (int t = 0; t < SUB; ++t) z[t] = b;
#pragma unroll 4
    for (int j = 0; j < a.r; ++j) {
        const float w = __ldg(a.w2 + (size_t)j * hd + c);
        const float4* y4 = (const float4*)(ys + j * SUB);
#pragma unroll
        for (int u = 0; u < SUB / 4; ++u) {
            const float4 y = y4[u];
            z[4 * u] = fmaf(w, y.x, z[4 * u]); z[4 * u + 1] = fmaf(w, y.y, z[4 * u + 1]);
            z[4 * u + 2] = fmaf(w, y.z, z[4 * u + 2]); z[4 * u + 3] = fmaf(w, y.w, z[4 * u + 3]);
        }
    }
    const float m = a.inv_tau * LOG2E;
    float s = 0.f;
#pragma unroll
    for (int t = 0; t < SUB; ++t) {
        s += log_sigmoid(z[t]) * m;
        if (t < n) L[(size_t)(r0 + t) * hd + c] = s;
    }
}

// ---------------------------------------------------------------- prompts: chunks
struct ChunkArgs {
    GlaArgs a;
    const float* L;                      // [T][H * D]
    float* ws;                           // [sequences][chunks][H][D * Dv + D]: update / starting state, then the chunk's decay
    int c_begin, chunks, slices, fuse;   // slices of value columns per head (at most SLICE_MAX each)
};
constexpr int SLICE_MAX = 128;

__host__ __device__ __forceinline__ int round4(int n) { return (n + 3) & ~3; }
__host__ __device__ __forceinline__ int slice_cols(int Dv, int slices) { return (round4(Dv) / 4 + slices - 1) / slices * 4; }
__device__ __forceinline__ size_t chunk_row(const ChunkArgs& c, int seq, int chunk, int h) {
    return (((size_t)seq * c.chunks + chunk) * c.a.H + h) * ((size_t)c.a.D * c.a.Dv + c.a.D);
}

// ROWS rows of `cols` columns at `src` into shared memory (row stride ls, a multiple of 4) by asynchronous copies, zeros from row nc /
// column cols on; a warp per row
template <int ROWS, int NT>
__device__ __forceinline__ void stage_rows(const float* src, size_t ld, int nc, int cols, float* dst, int ls, bool vec) {
    const int lane = threadIdx.x & 31;
    for (int r = threadIdx.x >> 5; r < ROWS; r += NT / 32) {
        const float* s = src + (size_t)r * ld;
        float* d = dst + r * ls;
        if (vec) {
            for (int c = lane * 4; c < ls; c += 128)
                if (r < nc && c < cols) cp_async16(d + c, s + c);
                else *(float4*)(d + c) = make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
            for (int c = lane; c < ls; c += 32)
                if (r < nc && c < cols) cp_async4(d + c, s + c);
                else d[c] = 0.f;
        }
    }
}

template <int MC>
__global__ void __launch_bounds__(256) gla_update_kernel(ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NS = MC / SUB;
    const GlaArgs& a = p.a;
    const int D = a.D, Dv = a.Dv, D8 = (D + 7) & ~7;
    const int h = blockIdx.z / p.slices, sl = blockIdx.z - h * p.slices;
    const int cw = slice_cols(Dv, p.slices), v0 = sl * cw, nv = min(cw, Dv - v0);
    float* Ks = sm;                      // [MC][D8], decayed to the chunk's end
    float* Vs = Ks + MC * D8;            // [MC][cw]
    float* Es = Vs + MC * cw;            // [NS][D8] sum of log2 decays from a sub-chunk's start to the chunk's end
    const int4 sq = a.seqs[blockIdx.y];
    const int c = p.c_begin + blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (c * MC >= sq.y || nv <= 0) return;
    const int nc = min(MC, sq.y - c * MC), r0 = sq.x + c * MC;
    const size_t hd = (size_t)a.H * D;
    stage_rows<MC, 256>(a.proj + (size_t)r0 * a.ld + a.v_off + (size_t)h * Dv + v0, a.ld, nc, nv, Vs, cw, a.vec);
    cp_async_commit();
    const float* Lh = p.L + (size_t)r0 * hd + (size_t)h * D;
    float* U = p.ws + chunk_row(p, blockIdx.y, blockIdx.x, h);
    for (int d = tid; d < D; d += 256) {
        float tot[NS], e = 0.f;
#pragma unroll
        for (int j = 0; j < NS; ++j) tot[j] = j * SUB < nc ? Lh[(size_t)min(nc - 1, j * SUB + SUB - 1) * hd + d] : 0.f;
#pragma unroll
        for (int j = NS - 1; j >= 0; --j) { e += tot[j]; Es[j * D8 + d] = e; }
        if (sl == 0) U[(size_t)D * Dv + d] = exp2_f(e);
    }
    __syncthreads();
    constexpr int B = 8;                                   // rows in flight per thread
    const float* kr = a.proj + (size_t)r0 * a.ld + a.k_off + (size_t)h * D;
    for (int d = lane; d < D8; d += 32)
        for (int s0 = warp; s0 < MC; s0 += 8 * B) {
            float kk[B], ll[B];
#pragma unroll
            for (int b = 0; b < B; ++b) {
                const int s = s0 + 8 * b;
                const bool in = s < nc && d < D;
                kk[b] = in ? kr[(size_t)s * a.ld + d] : 0.f;
                ll[b] = in ? Lh[(size_t)s * hd + d] : 0.f;
            }
#pragma unroll
            for (int b = 0; b < B; ++b) {
                const int s = s0 + 8 * b;
                if (s < MC) Ks[s * D8 + d] = s < nc && d < D ? kk[b] * exp2_f(Es[(s / SUB) * D8 + d] - ll[b]) : 0.f;
            }
        }
    cp_async_wait<0>();
    __syncthreads();
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
}

// scan over the chunks, one thread per state element
template <int MC>
__global__ void __launch_bounds__(256) gla_scan_kernel(ChunkArgs p) {
    const GlaArgs& a = p.a;
    const size_t mat = (size_t)a.D * a.Dv, per = mat + a.D, e = (size_t)blockIdx.x * 256 + threadIdx.x;
    const int h = blockIdx.y;
    const int4 sq = a.seqs[blockIdx.z];
    const int nchunks = (sq.y + MC - 1) / MC, n = min(nchunks, p.c_begin + p.chunks) - p.c_begin;
    if (n <= 0 || e >= mat) return;
    float* St = a.S + ((size_t)sq.z * a.H + h) * mat + e;
    float S = (sq.w > 0 || p.c_begin > 0) ? *St : 0.f;
    float* u = p.ws + chunk_row(p, blockIdx.z, 0, h) + e;
    const float* dc = p.ws + chunk_row(p, blockIdx.z, 0, h) + mat + e / a.Dv;
    const size_t step = (size_t)a.H * per;
    constexpr int B = 8;                                   // loads in flight per thread
    for (int c = 0; c < n; c += B) {
        float add[B], dec[B];
#pragma unroll
        for (int i = 0; i < B; ++i) {
            add[i] = c + i < n ? __ldcg(u + (size_t)(c + i) * step) : 0.f;
            dec[i] = c + i < n ? __ldg(dc + (size_t)(c + i) * step) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < B; ++i)
            if (c + i < n) {
                __stcg(u + (size_t)(c + i) * step, S);
                S = fmaf(S, dec[i], add[i]);
            }
    }
    *St = S;
}

// outputs of a chunk
constexpr int SLAB = 16;                 // state rows per slab

// A [D][MC] tile whose rows are permuted in groups of four elements, so that transposing stores and the products' loads (four
// neighbouring tokens of one channel, or sixteen of a channel and sixteen of the fourth one behind it) meet no bank conflicts
template <int MC> __device__ __forceinline__ int at_dt(int d, int t) {
    constexpr int M = MC / 4 < 8 ? MC / 4 - 1 : 7;
    return d * MC + (t ^ ((d & M) << 2));
}
// Weights of a chunk: one [SUB keys][SUB queries] block per pair of sub-chunks i >= j
__device__ __forceinline__ int at_st(int s, int t) {
    const int i = t / SUB, j = s / SUB;
    return ((i * (i + 1) / 2 + j) * SUB + s % SUB) * SUB + t % SUB;
}

// rows transposed into [D][MC]: a warp moves 8 consecutive elements of 4 rows at a time (whole sectors).  PAD: rows behind the last
// one repeat it inside its sub-chunk (running sums); otherwise they are zero.
template <int MC, int NT, bool PAD>
__device__ __forceinline__ void stage_transposed(const float* src, size_t ld, int nc, int D, float mult, float* dst) {
    constexpr int B = 8, NW = NT / 32;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, dl = lane & 7, tl = lane >> 3;
    const int last = (nc - 1) / SUB;
    for (int tg = warp; tg < MC / 4; tg += NW) {
        const int t = tg * 4 + tl;
        const bool in = t < nc || (PAD && t / SUB == last);
        const float* row = src + (size_t)min(t, nc - 1) * ld;
        for (int d0 = dl; d0 < D; d0 += 8 * B) {
            float r[B];
#pragma unroll
            for (int b = 0; b < B; ++b) r[b] = (in && d0 + 8 * b < D) ? __ldg(row + d0 + 8 * b) : 0.f;
#pragma unroll
            for (int b = 0; b < B; ++b)
                if (d0 + 8 * b < D) dst[at_dt<MC>(d0 + 8 * b, t)] = r[b] * mult;
        }
    }
}

template <int MC>
__global__ void __launch_bounds__(8 * MC, MC == 64 ? 2 : 1) gla_output_kernel(ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NT = 8 * MC, NS = MC / SUB, NP = NS * (NS - 1) / 2;
    const GlaArgs& a = p.a;
    const int D = a.D, Dv = a.Dv;
    const int h = blockIdx.z / p.slices, sl = blockIdx.z - h * p.slices;
    const int cw = slice_cols(Dv, p.slices), v0 = sl * cw, nv = min(cw, Dv - v0);
    float* Qt = sm;                      // [D][MC]
    float* R1 = Qt + D * MC;             // K transposed [D][MC], then V [MC][cw], then the outputs [MC][cw]
    float* Lt = R1 + MC * max(D, cw);    // [D][MC] running sums of log2 decays, then two slabs [SLAB][cw] of the starting state
    float* At = Lt + max(D * MC, 2 * SLAB * cw);           // [NP + NS][SUB][SUB]: weight of key s for query t
    float* Mb = At + (NP + NS) * SUB * SUB;                // [NP][D] decays over the sub-chunks between two
    const int4 sq = a.seqs[blockIdx.y];
    const int c = p.c_begin + blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (c * MC >= sq.y || nv <= 0) return;
    const int nc = min(MC, sq.y - c * MC), r0 = sq.x + c * MC;
    const bool has_state = sq.w > 0 || c > 0;
    const float* Sc = p.ws + chunk_row(p, blockIdx.y, blockIdx.x, h);
    const bool sv = a.vec && (D & 3) == 0;
    auto fetch_slab = [&](int b) {                         // slab b of the starting state
        stage_rows<SLAB, NT>(Sc + (size_t)b * SLAB * Dv + v0, Dv, min(SLAB, D - b * SLAB), nv, Lt + (b & 1) * SLAB * cw, cw, sv);
        cp_async_commit();
    };
    const float* rows = a.proj + (size_t)r0 * a.ld;
    const size_t hd = (size_t)a.H * D;
    stage_transposed<MC, NT, false>(rows + a.q_off + (size_t)h * D, a.ld, nc, D, a.q_scale, Qt);
    stage_transposed<MC, NT, false>(rows + a.k_off + (size_t)h * D, a.ld, nc, D, 1.f, R1);
    stage_transposed<MC, NT, true>(p.L + (size_t)r0 * hd + (size_t)h * D, hd, nc, D, 1.f, Lt);
    for (int i = tid; i < (NP + NS) * SUB * SUB; i += NT) At[i] = 0.f;
    __syncthreads();
    {   // weights inside a sub-chunk: four warps each, a warp takes four queries, a lane one key and every other group of four channels.
        // A key behind its query would give a positive exponent: such a pair's sum is thrown away.
        const int i = warp >> 2, tl = (warp & 3) * 4, s = lane & 15, half = lane >> 4;
        if (i * SUB + tl < nc) {
            const int t0 = i * SUB + tl, s0 = i * SUB + s;
            float acc[4] = {};
            for (int d0 = half * 4; d0 < D; d0 += 8) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int d = d0 + e;
                    if (d >= D) break;
                    const float k = R1[at_dt<MC>(d, s0)], l = Lt[at_dt<MC>(d, s0)];
                    const float4 q4 = *(const float4*)(Qt + at_dt<MC>(d, t0)), l4 = *(const float4*)(Lt + at_dt<MC>(d, t0));
                    acc[0] = fmaf(q4.x * k, exp2_f(l4.x - l), acc[0]);
                    acc[1] = fmaf(q4.y * k, exp2_f(l4.y - l), acc[1]);
                    acc[2] = fmaf(q4.z * k, exp2_f(l4.z - l), acc[2]);
                    acc[3] = fmaf(q4.w * k, exp2_f(l4.w - l), acc[3]);
                }
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float v = acc[e] + __shfl_xor_sync(0xffffffffu, acc[e], 16);
                if (half == 0 && s <= tl + e && t0 + e < nc) At[at_st(s0, t0 + e)] = v;
            }
        }
    }
    for (int pr = 0; pr < NP; ++pr) {                      // pair (i, j), i > j, at i (i - 1) / 2 + j
        int hi = 1, lo = pr;
        while (lo >= hi) { lo -= hi; ++hi; }
        for (int d = tid; d < D; d += NT) {
            float e = 0.f;
            for (int m = lo + 1; m < hi; ++m) e += Lt[at_dt<MC>(d, m * SUB + SUB - 1)];
            Mb[pr * D + d] = exp2_f(e);
        }
    }
    __syncthreads();
    for (int i = tid; i < D * MC; i += NT) {               // q decayed from its sub-chunk's start, k to its sub-chunk's end
        const int d = i / MC, t = i - d * MC, o = at_dt<MC>(d, t);
        const float l = Lt[o];
        Qt[o] *= exp2_f(l);
        R1[o] *= exp2_f(Lt[at_dt<MC>(d, (t / SUB) * SUB + SUB - 1)] - l);
    }
    __syncthreads();
    if (NP > 0) {   // weights between sub-chunks: 64 threads per pair, 2 queries x 2 keys each
        for (int w = tid; w < NP * 64; w += NT) {
            const int pr = w >> 6, x = w & 63;
            int hi = 1, lo = pr;
            while (lo >= hi) { lo -= hi; ++hi; }
            const int t0 = hi * SUB + (x >> 3) * 2, s0 = lo * SUB + (x & 7) * 2;
            if (t0 >= nc) continue;
            float a00 = 0.f, a01 = 0.f, a10 = 0.f, a11 = 0.f;
            const float* mp = Mb + pr * D;
#pragma unroll 8
            for (int d = 0; d < D; ++d) {
                const float2 q2 = *(const float2*)(Qt + at_dt<MC>(d, t0)), k2 = *(const float2*)(R1 + at_dt<MC>(d, s0));
                const float m = mp[d], kx = k2.x * m, ky = k2.y * m;
                a00 = fmaf(q2.x, kx, a00); a01 = fmaf(q2.x, ky, a01);
                a10 = fmaf(q2.y, kx, a10); a11 = fmaf(q2.y, ky, a11);
            }
            *(float2*)(At + at_st(s0, t0)) = make_float2(a00, a10);
            *(float2*)(At + at_st(s0 + 1, t0)) = make_float2(a01, a11);
        }
    }
    __syncthreads();                                       // K is done: V takes its place
    stage_rows<MC, NT>(rows + a.v_off + (size_t)h * Dv + v0, a.ld, nc, nv, R1, cw, a.vec);
    cp_async_commit();
    if (has_state) {
        if (NS > 1)                                        // q decayed from the chunk's start
            for (int i = tid; i < D * MC; i += NT) {
                const int d = i / MC, t = i - d * MC;
                if (t < SUB) continue;
                float e = 0.f;
                for (int m = 0; m < t / SUB; ++m) e += Lt[at_dt<MC>(d, m * SUB + SUB - 1)];
                Qt[at_dt<MC>(d, t)] *= exp2_f(e);
            }
        __syncthreads();                                   // the running sums are done: the state's slabs take their place
        fetch_slab(0);
    }
    const int nTv = cw / 4, ntiles = (MC / 4) * nTv;       // at most NT tiles of 4 tokens x 4 value columns
    const bool live = tid < ntiles;
    const int t0 = live ? (tid / nTv) * 4 : 0, w0 = live ? (tid % nTv) * 4 : 0;
    float acc[4][4] = {};
    cp_async_wait<0>();                                    // V and the first slab
    __syncthreads();
    if (has_state) {
        const int nslab = (D + SLAB - 1) / SLAB;
        for (int b = 0; b < nslab; ++b) {
            if (b + 1 < nslab) {                           // travels while this one is used
                fetch_slab(b + 1);
                if (b > 0) cp_async_wait<1>();
            } else {
                cp_async_wait<0>();
            }
            if (b > 0) __syncthreads();
            if (live) {
                const float* sb = Lt + (b & 1) * SLAB * cw + w0;
                const int ndd = min(SLAB, D - b * SLAB);
#pragma unroll 8
                for (int d = 0; d < ndd; ++d) {
                    const float4 q4 = *(const float4*)(Qt + at_dt<MC>(b * SLAB + d, t0)), s4 = *(const float4*)(sb + d * cw);
                    const float qq[4] = {q4.x, q4.y, q4.z, q4.w}, ssv[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i)
#pragma unroll
                        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(qq[i], ssv[j], acc[i][j]);
                }
            }
            __syncthreads();
        }
    }
    if (live) {
        const int send = min(nc, t0 + 4);
        const float* ar = At + at_st(0, t0);
        for (int j = 0; j * SUB < send; ++j) {             // one block of weights after the other
            const int ns = min(SUB, send - j * SUB);
            const float* vr = R1 + j * SUB * cw + w0;
#pragma unroll 4
            for (int s = 0; s < ns; ++s) {
                const float4 aa = *(const float4*)(ar + (j * SUB + s) * SUB), v4 = *(const float4*)(vr + s * cw);
                const float ww[4] = {aa.x, aa.y, aa.z, aa.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int k = 0; k < 4; ++k) acc[i][k] = fmaf(ww[i], vv[k], acc[i][k]);
            }
        }
    }
    __syncthreads();                                       // V is done: the outputs take its place
    if (live)
#pragma unroll
        for (int i = 0; i < 4; ++i) *(float4*)(R1 + (t0 + i) * cw + w0) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    __syncthreads();
    for (int t = warp; t < nc; t += NT / 32) {             // a warp per row: norm, weight, gate (or the plain output)
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
        for (int v = lane; v < nv; v += 32) dst[v] = o[v] * inv * a.w[h * Dv + v] * silu_f(gr[v]);
    }
}

inline bool mult4(long long v) { return (v & 3) == 0; }
inline bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

template <int VW>
int launch_step(const GlaArgs& a, int n_seqs, int blocks, int slice, cudaStream_t st) {
    const size_t smem = sizeof(float) * (3 * (size_t)round4(a.D) + (size_t)ST * VW + (size_t)slice + 4);
    PGK_REQUIRE(smem <= 200 * 1024, "seq_gla_step failed: heads of %d x %d need %zu bytes of shared memory", a.D, a.Dv, smem);
    static bool configured = false;
    if (smem > 40 * 1024 && !configured) {
        PGK_CUDA(cudaFuncSetAttribute(gla_step_kernel<VW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
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
    PGK_CUDA(cudaLaunchKernelEx(&cfg, gla_step_kernel<VW>, a, slice));
    return 0;
}

constexpr size_t CHUNK_SMEM = 224 * 1024;

size_t output_smem(int MC, int D, int cw) {
    const size_t ns = MC / SUB, np = ns * (ns - 1) / 2, dm = (size_t)D * MC, vm = (size_t)MC * cw, sl = 2 * (size_t)SLAB * cw;
    return sizeof(float) * (dm + (dm > vm ? dm : vm) + (dm > sl ? dm : sl) + (np + ns) * SUB * SUB + np * D);
}
int value_slices(int vdim) { return (vdim + SLICE_MAX - 1) / SLICE_MAX; }
// tokens per chunk: what fits a block's shared memory (0: keys too large)
int chunk_tokens(int D, int Dv) {
    const int cw = slice_cols(Dv, value_slices(Dv));
    for (int mc : {64, 32, 16})
        if (output_smem(mc, D, cw) <= CHUNK_SMEM) return mc;
    return 0;
}

template <int MC>
int launch_chunks(ChunkArgs& p, int n_seqs, cudaStream_t st) {
    const GlaArgs& a = p.a;
    const int cw = slice_cols(a.Dv, p.slices), D8 = (a.D + 7) & ~7;
    const size_t smem_u = sizeof(float) * ((size_t)MC * D8 + (size_t)MC * cw + (size_t)(MC / SUB) * D8), smem_o = output_smem(MC, a.D, cw);
    static bool configured = false;
    if (!configured) {
        PGK_CUDA(cudaFuncSetAttribute(gla_update_kernel<MC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)CHUNK_SMEM));
        PGK_CUDA(cudaFuncSetAttribute(gla_output_kernel<MC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)CHUNK_SMEM));
        configured = true;
    }
    const dim3 grid(p.chunks, n_seqs, a.H * p.slices);
    PGK_CUDA(launch(gla_update_kernel<MC>, grid, dim3(256), smem_u, st, p));
    const size_t mat = (size_t)a.D * a.Dv;
    PGK_CUDA(launch(gla_scan_kernel<MC>, dim3((unsigned)((mat + 255) / 256), a.H, n_seqs), dim3(256), 0, st, p));
    PGK_CUDA(launch(gla_output_kernel<MC>, grid, dim3(8 * MC), smem_o, st, p));
    return 0;
}

int fill_args(GlaArgs& a, const char* who, const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, int y_off, int r,
              const float* w2, const float* b2, float inv_tau, float q_scale, const float* weight, float eps, float* out, int ldo,
              float* S, const int32_t* seqs, int heads, int dim, int vdim) {
    PGK_REQUIRE(heads > 0 && dim > 0 && vdim > 0 && r > 0, "%s failed: %d heads of %d x %d, inner size %d", who, heads, dim, vdim, r);
    PGK_REQUIRE(proj && w2 && b2 && weight && out && S && seqs, "%s failed: a missing operand", who);
    a = GlaArgs{proj, ld, q_off, k_off, v_off, g_off, y_off, w2, b2, r, inv_tau, q_scale, weight, eps, out, ldo, S, (const int4*)seqs,
                heads, dim, vdim, 0};
    a.vec = mult4(ld) && mult4(v_off) && mult4(vdim) && aligned16(proj) && aligned16(S);
    return 0;
}

}  // namespace

extern "C" {

int pgk_seq_gla_chunk_tokens(int dim, int vdim) { return chunk_tokens(dim, vdim); }

int pgk_seq_gla_fused_finish(int vdim) { return value_slices(vdim) == 1 ? 1 : 0; }

int pgk_seq_gla_step(const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, int y_off, int inner, const float* w2,
                     const float* b2, float inv_tau, float q_scale, const float* weight, float eps, float* out, int ldo, float* S,
                     const int32_t* seqs, int n_seqs, int heads, int dim, int vdim, void* stream) {
    GlaArgs a;
    if (fill_args(a, "seq_gla_step", proj, ld, q_off, k_off, v_off, g_off, y_off, inner, w2, b2, inv_tau, q_scale, weight, eps, out, ldo,
                  S, seqs, heads, dim, vdim)) return 1;
    if (n_seqs <= 0) return 0;
    // value columns are cut over a cluster until the grid fills the GPU, never into slices of fewer than 16
    int blocks = 1;
    while (blocks < 8 && (long long)n_seqs * heads * blocks < 148 && vdim / (2 * blocks) >= 16) blocks *= 2;
    const int slice = ((vdim + blocks - 1) / blocks + 3) & ~3;
    return mult4(vdim) && aligned16(S) ? launch_step<4>(a, n_seqs, blocks, slice, (cudaStream_t)stream)
                                       : launch_step<1>(a, n_seqs, blocks, slice, (cudaStream_t)stream);
}

/* L: [tokens][heads * dim] floats */
int pgk_seq_gla_decays(const float* proj, int ld, int y_off, int inner, const float* w2, const float* b2, float inv_tau,
                       const int32_t* seqs, int n_seqs, int max_rows, int heads, int dim, float* L, void* stream) {
    PGK_REQUIRE(heads > 0 && dim > 0 && inner > 0 && inner <= 512 && w2 && b2 && L, "seq_gla_decays failed: %d heads of %d, inner size %d", heads, dim, inner);
    if (n_seqs <= 0 || max_rows <= 0) return 0;
    GlaArgs a{};
    a.proj = proj; a.ld = ld; a.y_off = y_off; a.r = inner; a.w2 = w2; a.b2 = b2; a.inv_tau = inv_tau; a.seqs = (const int4*)seqs;
    a.H = heads; a.D = dim;
    PGK_CUDA(launch(gla_decays_kernel, dim3((max_rows + SUB - 1) / SUB, (heads * dim + 255) / 256, n_seqs), dim3(256),
                    (size_t)inner * SUB * sizeof(float), (cudaStream_t)stream, a, L));
    return 0;
}

int pgk_seq_gla_chunks(const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, const float* L, float q_scale,
                       const float* weight, float eps, float* out, int ldo, float* S, const int32_t* seqs, int n_seqs, int heads, int dim,
                       int vdim, int chunk_begin, int chunks, float* workspace, void* stream) {
    ChunkArgs p{};
    if (fill_args(p.a, "seq_gla_chunks", proj, ld, q_off, k_off, v_off, g_off, 0, 1, L, L, 1.f, q_scale, weight, eps, out, ldo, S, seqs,
                  heads, dim, vdim)) return 1;
    PGK_REQUIRE(L && workspace && chunk_begin >= 0, "seq_gla_chunks failed: a missing workspace");
    const int mc = chunk_tokens(dim, vdim);
    PGK_REQUIRE(mc > 0, "seq_gla_chunks failed: keys of %d do not fit shared memory", dim);
    if (n_seqs <= 0 || chunks <= 0) return 0;
    p.a.vec = p.a.vec && aligned16(workspace);
    p.L = L; p.ws = workspace; p.c_begin = chunk_begin; p.chunks = chunks;
    p.slices = value_slices(vdim);
    p.fuse = p.slices == 1;
    if (mc == 64) return launch_chunks<64>(p, n_seqs, (cudaStream_t)stream);
    if (mc == 32) return launch_chunks<32>(p, n_seqs, (cudaStream_t)stream);
    return launch_chunks<16>(p, n_seqs, (cudaStream_t)stream);
}

}  // extern "C"
