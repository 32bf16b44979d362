// The state recurrences of state_mixers.cu for long portions of prompts, in chunks of 64 tokens on the tensor cores
// instead of token by token: per (sequence, head) a float32 state S [rows, columns] with
//   gated write   S = diag(exp(g)) S + k v^T,         o = q_scale S^T q              (g: log decay of every row)
//   head decay    S = exp(g) S + beta k v^T,          o = q_scale S^T q + skip v     (g, beta: one number per head)
// Three kernels:
//   1. chunk_state: what a chunk alone adds to the state by its end, U = sum_j decay(j -> end) k_j v_j^T, and its decay;
//   2. chunk_scan: S before every chunk, chunk by chunk, and the request's state after the last one;
//   3. chunk_output: o_i = decay(start -> i) q_i S + sum_(j <= i) A_ij v_j, A_ij = q_i . (decay(j -> i) k_j).
// Matrix products run as m16n8k8 TF32 products of operands split in two TF32 terms each (x = hi + lo; hi hi + hi lo + lo hi,
// float32 accumulation), which keeps about 21 bits of every product: the float32 arithmetic of the walk within rounding.
// Every decay factor is the exponential of a sum of log decays between two tokens, so none exceeds one: for the gated
// write the factor exp(b_i - b_j) of a row is taken apart at the borders of blocks of 16 tokens that lie between j and i,
// and inside a block it is evaluated pair by pair.
#include "mma_helpers.cuh"
#include <math.h>

namespace {
constexpr int CHUNK = 64;
constexpr int COLS = 128;                 // columns a CTA takes: of one head, or of two whole heads that share q and k
constexpr int BLOCK = 16;
constexpr int VP = COLS + 8;              // pitch of the staged values: fragment reads without bank conflicts
constexpr int AP = CHUNK + 4;             // pitch of the chunk's token x token matrix
constexpr float LOG2E = 1.4426950408889634f;
constexpr int MAX_HP = 2;

enum Form : int { GATED = 0, HEAD = 2 };  // the codes of rs_state_recurrence

struct ChunkParams {
    const float* q; long q_stride;        // [T, (heads / group) * rows]
    const float* k; long k_stride;
    const float* g; long g_stride;        // log decays: gated write [T, heads * rows], head decay [T, heads]
    const float* beta; long beta_stride;  // [T, heads], head decay only
    const float* v; long v_stride;        // [T, heads * columns]
    float* out; long out_stride;
    float* state; long state_stride;      // [slots, heads * columns * padded rows], a head column by column
    const int* q_start; const int* slots;
    const int* chunk_seq; const int* chunk_start; const int* seq_first_chunk;
    float* sums;                          // [chunks, heads, columns, padded rows]: U, then S before the chunk
    float* decays;                        // [chunks, heads, padded rows] (gated) or [chunks, heads]
    int heads, group, columns, rows, hp, col_tiles;
    float q_scale; const float* skip;
};

__device__ __forceinline__ float exp_of(float x) { return fast_exp2(x * LOG2E); }

__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;                   // the leading 10 bits of the mantissa, then the next ones
    lo = __float_as_uint(x - __uint_as_float(hi)) & 0xffffe000u;
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct AFrag { uint32_t hi[4], lo[4]; };
__device__ __forceinline__ void make_a(AFrag& f, float a0, float a1, float a2, float a3) {
    split_tf32(a0, f.hi[0], f.lo[0]); split_tf32(a1, f.hi[1], f.lo[1]);
    split_tf32(a2, f.hi[2], f.lo[2]); split_tf32(a3, f.hi[3], f.lo[3]);
}
struct BFrag { uint32_t h0, l0, h1, l1; };
__device__ __forceinline__ BFrag make_b(float b0, float b1) {
    BFrag f;
    split_tf32(b0, f.h0, f.l0);
    split_tf32(b1, f.h1, f.l1);
    return f;
}
__device__ __forceinline__ void mma_split(float (&d)[4], const AFrag& a, const BFrag& b) {
    mma_tf32(d, a.lo, b.h0, b.h1);
    mma_tf32(d, a.hi, b.l0, b.l1);
    mma_tf32(d, a.hi, b.h0, b.h1);
}
// the same for two blocks of rows: two products of one sum do not follow each other directly
__device__ __forceinline__ void mma_split2(float (&d0)[4], float (&d1)[4], const AFrag& a0, const AFrag& a1, const BFrag& b) {
    mma_tf32(d0, a0.lo, b.h0, b.h1); mma_tf32(d1, a1.lo, b.h0, b.h1);
    mma_tf32(d0, a0.hi, b.l0, b.l1); mma_tf32(d1, a1.hi, b.l0, b.l1);
    mma_tf32(d0, a0.hi, b.h0, b.h1); mma_tf32(d1, a1.hi, b.h0, b.h1);
}

struct Place { int s, t0, nt, h0, qk, col0, ncols; };       // of a CTA: sequence, first token row, tokens, heads, columns
__device__ __forceinline__ Place place_of(const ChunkParams& p) {
    Place c;
    const int ch = blockIdx.x;
    c.s = p.chunk_seq[ch];
    const int start = p.chunk_start[ch];
    c.t0 = p.q_start[c.s] + start;
    c.nt = min(CHUNK, p.q_start[c.s + 1] - c.t0);
    const int unit = blockIdx.y / p.col_tiles, tile = blockIdx.y % p.col_tiles;
    c.h0 = unit * p.hp;
    c.qk = c.h0 / p.group;
    c.col0 = tile * COLS;                                   // nonzero only with one head per CTA
    c.ncols = p.hp > 1 ? p.hp * p.columns : min(COLS, p.columns - c.col0);
    return c;
}
// Staged column cc is column (first_column + cc) of the row that all heads' columns make; which of the CTA's heads it is of:
__device__ __forceinline__ size_t first_column(const ChunkParams& p, const Place& c) { return (size_t)c.h0 * p.columns + c.col0; }
__device__ __forceinline__ int head_of(const ChunkParams& p, int cc) { return p.hp > 1 && cc >= p.columns ? 1 : 0; }

// values of the CTA's columns, zero beyond the chunk's tokens and the columns (asynchronous copies where rows are aligned)
template <int THREADS>
__device__ __forceinline__ void stage_values(const ChunkParams& p, const Place& c, float* Vs) {
    const float* v = p.v + (size_t)c.t0 * p.v_stride + (size_t)c.h0 * p.columns + c.col0;
    const bool aligned = ((uintptr_t)v & 15) == 0 && p.v_stride % 4 == 0;
#pragma unroll 4
    for (int i = threadIdx.x; i < CHUNK * (COLS / 4); i += THREADS) {
        const int j = i / (COLS / 4), cc = (i % (COLS / 4)) * 4;
        const float* src = v + (size_t)j * p.v_stride + cc;
        float* dst = Vs + j * VP + cc;
        if (aligned && j < c.nt && cc + 3 < c.ncols) {
            cp_async16(smem_addr(dst), src);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) dst[e] = j < c.nt && cc + e < c.ncols ? src[e] : 0.f;
        }
    }
}

// Rows of RP values with 16-byte fragment reads: row r's halves of 32 values trade places when bit 0 of r ^ (r >> 1) is
// set, so that neither rows r, r + 1 nor rows r, r + 2 side by side meet in a bank.
__device__ __forceinline__ int turned(int r) { return ((r ^ (r >> 1)) & 1) << 4; }

// rows of q, k or g of one head: [CHUNK][RP] turned, zero beyond the chunk's tokens and the head's rows
template <int RP, int THREADS>
__device__ __forceinline__ void stage_rows(const float* src, long stride, float* dst, int nt, int rows) {
#pragma unroll 4
    for (int i = threadIdx.x; i < CHUNK * (RP / 4); i += THREADS) {
        const int j = i / (RP / 4), d = (i % (RP / 4)) * 4;
        float* to = dst + j * RP + (d ^ turned(j));
        if (j < nt && d < rows) cp_async16(smem_addr(to), src + (size_t)j * stride + d);
        else *reinterpret_cast<float4*>(to) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
}

// ------------------------------------------------------------------------------------------------ 1: a chunk alone
template <int FORM, int RP>
__global__ void __launch_bounds__(256) chunk_state_kernel(ChunkParams p) {
    constexpr int KP = RP + 8, SEGS = 256 / RP, SEG = CHUNK / SEGS;
    extern __shared__ __align__(16) float smem[];
    float* Ks = smem;                                        // [CHUNK][KP]
    float* Vs = Ks + CHUNK * KP;                             // [CHUNK][VP]
    float (*scale)[CHUNK] = reinterpret_cast<float (*)[CHUNK]>(Vs + CHUNK * VP);      // head decay: [HP][CHUNK]
    float* part = Vs + CHUNK * VP;                           // gated: [SEGS][RP]
    (void)scale; (void)part;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
    const Place c = place_of(p);
    stage_values<256>(p, c, Vs);
    if (FORM == GATED) {
        const int d = tid % RP, seg = tid / RP;
        const bool live = d < p.rows;
        const float* g = p.g + (size_t)c.t0 * p.g_stride + (size_t)c.h0 * p.rows + d;
        const float* k = p.k + (size_t)c.t0 * p.k_stride + (size_t)c.qk * p.rows + d;
        float gv[SEG], kv[SEG], sum = 0.f;
#pragma unroll
        for (int e = 0; e < SEG; ++e) {
            const int j = seg * SEG + e;
            const bool on = live && j < c.nt;
            gv[e] = on ? g[(size_t)j * p.g_stride] : 0.f;
            kv[e] = on ? k[(size_t)j * p.k_stride] : 0.f;
        }
#pragma unroll
        for (int e = 0; e < SEG; ++e) sum += gv[e];
        part[seg * RP + d] = sum;
        __syncthreads();
        float suffix = 0.f;                                  // log decay from token j to the chunk's end
        for (int e = SEGS - 1; e > seg; --e) suffix += part[e * RP + d];
#pragma unroll
        for (int e = SEG - 1; e >= 0; --e) {
            Ks[(seg * SEG + e) * KP + d] = kv[e] * exp_of(suffix);
            suffix += gv[e];
        }
        if (seg == 0 && c.col0 == 0) p.decays[((size_t)blockIdx.x * p.heads + c.h0) * RP + d] = live ? exp_of(suffix) : 0.f;
    } else {
        const float* k = p.k + (size_t)c.t0 * p.k_stride + (size_t)c.qk * p.rows;
#pragma unroll 4
        for (int i = tid; i < CHUNK * (RP / 4); i += 256) {
            const int j = i / (RP / 4), d = (i % (RP / 4)) * 4;
            if (j < c.nt && d < p.rows) cp_async16(smem_addr(Ks + j * KP + d), k + (size_t)j * p.k_stride + d);
            else *reinterpret_cast<float4*>(Ks + j * KP + d) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
        // per head: beta_j times the decay from j to the end, by a scan from the end (two tokens a lane)
        for (int hh = warp; hh < p.hp; hh += 8) {
            const int h = c.h0 + hh, j0 = 2 * lane, j1 = j0 + 1;
            const float* g = p.g + (size_t)c.t0 * p.g_stride + h;
            const float* b = p.beta + (size_t)c.t0 * p.beta_stride + h;
            const float g0 = j0 < c.nt ? g[(size_t)j0 * p.g_stride] : 0.f, g1 = j1 < c.nt ? g[(size_t)j1 * p.g_stride] : 0.f;
            float incl = g0 + g1;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_down_sync(0xffffffffu, incl, o);
                if (lane + o < 32) incl += up;
            }
            float after = __shfl_down_sync(0xffffffffu, incl, 1);                         // log decay after this lane's tokens
            if (lane == 31) after = 0.f;
            scale[hh][j1] = j1 < c.nt ? b[(size_t)j1 * p.beta_stride] * exp_of(after) : 0.f;
            scale[hh][j0] = j0 < c.nt ? b[(size_t)j0 * p.beta_stride] * exp_of(after + g1) : 0.f;
            if (lane == 0 && c.col0 == 0) p.decays[(size_t)blockIdx.x * p.heads + h] = exp_of(incl);
        }
    }
    cp_async_wait_all();
    __syncthreads();
    // U = K^T V: a warp takes 32 rows of the state and COLS / CP columns
    constexpr int PAIRS = RP / 32, CP = PAIRS >= 4 ? 2 : 8 / PAIRS, NBW = COLS / 8 / CP;
    const int n_base = (warp % CP) * NBW * 8;
    for (int pair = warp / CP; pair < PAIRS; pair += 8 / CP) {
        float acc[2][NBW][4];
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int nb = 0; nb < NBW; ++nb)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[m][nb][e] = 0.f;
        const int ksteps = (c.nt + 7) / 8;
        for (int ks = 0; ks < ksteps; ++ks) {
            const float* r0 = Ks + (ks * 8 + tig) * KP + pair * 32 + gid;
            const float* r1 = r0 + 4 * KP;
            AFrag a[2];
#pragma unroll
            for (int m = 0; m < 2; ++m) make_a(a[m], r0[16 * m], r0[16 * m + 8], r1[16 * m], r1[16 * m + 8]);
#pragma unroll
            for (int nb = 0; nb < NBW; ++nb) {
                const int n = n_base + nb * 8;
                if (n >= c.ncols) continue;
                const float* vb = Vs + (ks * 8 + tig) * VP + n + gid;
                float v0 = vb[0], v1 = vb[4 * VP];
                if (FORM == HEAD) {
                    const float* sc = scale[head_of(p, n)];
                    v0 *= sc[ks * 8 + tig]; v1 *= sc[ks * 8 + tig + 4];
                }
                const BFrag b = make_b(v0, v1);
                mma_split2(acc[0][nb], acc[1][nb], a[0], a[1], b);
            }
        }
#pragma unroll
        for (int nb = 0; nb < NBW; ++nb)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int cc = n_base + nb * 8 + 2 * tig + e;
                if (cc >= c.ncols) continue;
                float* u = p.sums + ((size_t)blockIdx.x * p.heads * p.columns + first_column(p, c) + cc) * RP + pair * 32 + gid;
#pragma unroll
                for (int m = 0; m < 2; ++m) { u[16 * m] = acc[m][nb][e]; u[16 * m + 8] = acc[m][nb][e + 2]; }
            }
    }
}

// ------------------------------------------------------------------------------------------------ 2: from chunk to chunk
// A thread per four rows of a column of a head's state.
template <int FORM>
__global__ void __launch_bounds__(256) chunk_scan_kernel(ChunkParams p, int rp) {
    const int i = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y, s = blockIdx.z;
    const int per_col = rp / 4;
    if (i >= p.columns * per_col) return;
    const int r = (i % per_col) * 4;
    const size_t at = (size_t)h * p.columns * rp + (size_t)i * 4, step = (size_t)p.heads * p.columns * rp;
    float* state = p.state + (size_t)p.slots[s] * p.state_stride + at;
    float4 S = *reinterpret_cast<const float4*>(state);
    const int c0 = p.seq_first_chunk[s], c1 = p.seq_first_chunk[s + 1];
    constexpr int AHEAD = 4;
    for (int c = c0; c < c1; c += AHEAD) {
        float4 U[AHEAD], D[AHEAD];
#pragma unroll
        for (int e = 0; e < AHEAD; ++e) {
            const int cc = min(c + e, c1 - 1);
            U[e] = __ldcg(reinterpret_cast<const float4*>(p.sums + (size_t)cc * step + at));
            if (FORM == GATED) D[e] = __ldg(reinterpret_cast<const float4*>(p.decays + ((size_t)cc * p.heads + h) * rp + r));
            else { const float d = __ldg(p.decays + (size_t)cc * p.heads + h); D[e] = make_float4(d, d, d, d); }
        }
#pragma unroll
        for (int e = 0; e < AHEAD; ++e) {
            if (c + e >= c1) break;
            *reinterpret_cast<float4*>(p.sums + (size_t)(c + e) * step + at) = S;
            S.x = fmaf(D[e].x, S.x, U[e].x); S.y = fmaf(D[e].y, S.y, U[e].y);
            S.z = fmaf(D[e].z, S.z, U[e].z); S.w = fmaf(D[e].w, S.w, U[e].w);
        }
    }
    *reinterpret_cast<float4*>(state) = S;
}

// ------------------------------------------------------------------------------------------------ 3: the outputs
template <int FORM, int RP>
struct OutputLayout {
    static constexpr int P = RP;                             // pitch of q, k, g and the state's columns (turned rows)
    static constexpr int A_HEADS = FORM == GATED ? 1 : MAX_HP;
    static constexpr size_t q = 0, k = q + CHUNK * P, s = k + CHUNK * P, v = s + COLS * P, a = v + CHUNK * VP,
                            x = a + A_HEADS * CHUNK * AP;
    // gated: g [CHUNK][P], block decays [4][RP], decays up to a block [4][RP]; head decay: cumulative log decay in two
    // terms, and strength
    static constexpr size_t total = FORM == GATED ? x + CHUNK * P + 8 * RP : x + 3 * MAX_HP * CHUNK;
};

// a 16 x 8 block of q k^T (rows of q from ri, rows of k from rj), q times f0[d] f1[d] if given
template <int RP>
__device__ __forceinline__ void token_block(const float* Q, const float* K, int ri, int rj, const float* f0, const float* f1, int gid,
                                            int tig, float (&acc)[4]) {
    acc[0] = acc[1] = acc[2] = acc[3] = 0.f;
    const float *qa = Q + (ri + gid) * RP, *qb = qa + 8 * RP, *kb = K + (rj + gid) * RP;
    const int qt = turned(ri + gid), kt = turned(rj + gid);          // rows eight apart are turned alike
#pragma unroll 4
    for (int d0 = 0; d0 < RP; d0 += 16) {
        const int d = d0 + 4 * tig;
        float4 x = *reinterpret_cast<const float4*>(qa + (d ^ qt)), y = *reinterpret_cast<const float4*>(qb + (d ^ qt));
        const float4 z = *reinterpret_cast<const float4*>(kb + (d ^ kt));
        if (f0) {
            const float4 f = *reinterpret_cast<const float4*>(f0 + d);
            x.x *= f.x; x.y *= f.y; x.z *= f.z; x.w *= f.w;
            y.x *= f.x; y.y *= f.y; y.z *= f.z; y.w *= f.w;
        }
        if (f1) {
            const float4 f = *reinterpret_cast<const float4*>(f1 + d);
            x.x *= f.x; x.y *= f.y; x.z *= f.z; x.w *= f.w;
            y.x *= f.x; y.y *= f.y; y.z *= f.z; y.w *= f.w;
        }
        AFrag a;
        make_a(a, x.x, y.x, x.y, y.y);                       // the sixteen coordinates in the order 4 tig + e, for both operands
        mma_split(acc, a, make_b(z.x, z.y));
        make_a(a, x.z, y.z, x.w, y.w);
        mma_split(acc, a, make_b(z.z, z.w));
    }
}

template <int FORM, int RP>
__global__ void __launch_bounds__(512, 1) chunk_output_kernel(ChunkParams p) {
    using L = OutputLayout<FORM, RP>;
    constexpr int P = L::P;
    static_assert(P == RP, "turned rows have no pad");
    extern __shared__ __align__(16) float smem[];
    float *Q = smem + L::q, *K = smem + L::k, *Ss = smem + L::s, *Vs = smem + L::v, *A = smem + L::a;
    float* G = smem + L::x;                                  // gated
    float *Pb = G + CHUNK * P, *E = Pb + 4 * RP;
    float (*bc)[CHUNK] = reinterpret_cast<float (*)[CHUNK]>(smem + L::x);                       // head decay
    float (*bl)[CHUNK] = bc + MAX_HP, (*wt)[CHUNK] = bl + MAX_HP;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
    const Place c = place_of(p);
    stage_rows<RP, 512>(p.q + (size_t)c.t0 * p.q_stride + (size_t)c.qk * p.rows, p.q_stride, Q, c.nt, p.rows);
    stage_rows<RP, 512>(p.k + (size_t)c.t0 * p.k_stride + (size_t)c.qk * p.rows, p.k_stride, K, c.nt, p.rows);
    if (FORM == GATED) stage_rows<RP, 512>(p.g + (size_t)c.t0 * p.g_stride + (size_t)c.h0 * p.rows, p.g_stride, G, c.nt, p.rows);
    cp_async_commit();
    // the values and the state before the chunk are asked for now and needed last
    stage_values<512>(p, c, Vs);
#pragma unroll 4
    for (int i = tid; i < COLS * (RP / 4); i += 512) {
        const int cc = i / (RP / 4), d = (i % (RP / 4)) * 4;
        if (cc < c.ncols)
            cp_async16(smem_addr(Ss + cc * P + (d ^ turned(cc))),
                       p.sums + ((size_t)blockIdx.x * p.heads * p.columns + first_column(p, c) + cc) * RP + d);
    }
    cp_async_commit();
    if (FORM == HEAD) {
        for (int hh = warp; hh < p.hp; hh += 16) {
            const int h = c.h0 + hh, j0 = 2 * lane, j1 = j0 + 1;
            const float* g = p.g + (size_t)c.t0 * p.g_stride + h;
            const float* b = p.beta + (size_t)c.t0 * p.beta_stride + h;
            const float g0 = j0 < c.nt ? g[(size_t)j0 * p.g_stride] : 0.f, g1 = j1 < c.nt ? g[(size_t)j1 * p.g_stride] : 0.f;
            // summed in float64 and kept in two terms: a difference of two sums is then as exact as the log decays are
            double incl = (double)g0 + (double)g1;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double up = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += up;
            }
            const double b0 = incl - (double)g1;
            bc[hh][j0] = (float)b0; bc[hh][j1] = (float)incl;
            bl[hh][j0] = (float)(b0 - (double)(float)b0); bl[hh][j1] = (float)(incl - (double)(float)incl);
            wt[hh][j0] = j0 < c.nt ? b[(size_t)j0 * p.beta_stride] : 0.f;
            wt[hh][j1] = j1 < c.nt ? b[(size_t)j1 * p.beta_stride] : 0.f;
        }
    }
    cp_async_wait<1>();
    __syncthreads();
    if (FORM == GATED) {
        // running log decay inside every block of 16 tokens, and the block's decay
        for (int i = tid; i < 4 * RP; i += 512) {
            const int d = i % RP, blk = i / RP;
            float b = 0.f;
#pragma unroll
            for (int j = 0; j < BLOCK; ++j) {
                float* gj = G + (blk * BLOCK + j) * P + (d ^ turned(j));      // a block's first row is turned like row 0
                b += *gj;
                *gj = b;
            }
            Pb[blk * RP + d] = exp_of(b);
        }
        __syncthreads();
        for (int i = tid; i < RP; i += 512) {
            float e = 1.f;
#pragma unroll
            for (int blk = 0; blk < 4; ++blk) { E[blk * RP + i] = e; e *= Pb[blk * RP + i]; }
        }
        // pairs of tokens inside a block: 2 x 2 of them and a quarter of the rows per thread
        for (int i = tid; i < 4 * 36 * 4; i += 512) {        // 4 blocks, 36 of their 8 x 8 pairs of pairs, 4 lanes each
            const int part = i & 3, blk = (i >> 2) / 36;
            int t = (i >> 2) % 36, ti = 0;
            while (t > ti) { t -= ti + 1; ++ti; }            // row ti of the triangle holds ti + 1 of them
            const int r0 = blk * BLOCK + 2 * ti, s0 = blk * BLOCK + 2 * t;
            const float *q0 = Q + r0 * P, *q1 = q0 + P, *k0 = K + s0 * P, *k1 = k0 + P;
            const float *bq0 = G + r0 * P, *bq1 = bq0 + P, *bk0 = G + s0 * P, *bk1 = bk0 + P;
            float s00 = 0.f, s01 = 0.f, s10 = 0.f, s11 = 0.f;
            const int u0 = turned(r0), u1 = turned(r0 + 1), w0 = turned(s0), w1 = turned(s0 + 1);
            for (int d = 4 * part; d < RP; d += 16) {
                const float4 x0 = *reinterpret_cast<const float4*>(q0 + (d ^ u0)), x1 = *reinterpret_cast<const float4*>(q1 + (d ^ u1));
                const float4 y0 = *reinterpret_cast<const float4*>(k0 + (d ^ w0)), y1 = *reinterpret_cast<const float4*>(k1 + (d ^ w1));
                const float4 a0 = *reinterpret_cast<const float4*>(bq0 + (d ^ u0)), a1 = *reinterpret_cast<const float4*>(bq1 + (d ^ u1));
                const float4 c0 = *reinterpret_cast<const float4*>(bk0 + (d ^ w0)), c1 = *reinterpret_cast<const float4*>(bk1 + (d ^ w1));
#define RS_PAIRS(e)                                                                                                             \
                s00 = fmaf(x0.e * y0.e, exp_of(a0.e - c0.e), s00); s10 = fmaf(x1.e * y0.e, exp_of(a1.e - c0.e), s10);           \
                s01 = fmaf(x0.e * y1.e, exp_of(fminf(a0.e - c1.e, 0.f)), s01); s11 = fmaf(x1.e * y1.e, exp_of(a1.e - c1.e), s11);
                RS_PAIRS(x) RS_PAIRS(y) RS_PAIRS(z) RS_PAIRS(w)
#undef RS_PAIRS
            }
#pragma unroll
            for (int o = 1; o < 4; o <<= 1) {
                s00 += __shfl_xor_sync(0xffffffffu, s00, o); s01 += __shfl_xor_sync(0xffffffffu, s01, o);
                s10 += __shfl_xor_sync(0xffffffffu, s10, o); s11 += __shfl_xor_sync(0xffffffffu, s11, o);
            }
            if (part == 0) {
                A[r0 * AP + s0] = s00; A[(r0 + 1) * AP + s0] = s10;
                A[r0 * AP + s0 + 1] = ti == t ? 0.f : s01;   // on the diagonal the upper right pair looks ahead
                A[(r0 + 1) * AP + s0 + 1] = s11;
                if (ti != t) {                               // the mirror image lies above the diagonal
                    A[s0 * AP + r0] = A[s0 * AP + r0 + 1] = A[(s0 + 1) * AP + r0] = A[(s0 + 1) * AP + r0 + 1] = 0.f;
                }
            }
        }
        __syncthreads();
        // q by its decay since its block's start, k by its decay to its block's end
        for (int i = tid; i < CHUNK * RP; i += 512) {
            const int j = i / RP, d = i % RP;
            const int last = j | (BLOCK - 1), at = j * P + (d ^ turned(j));
            const float b = G[at], end = G[last * P + (d ^ turned(last))];
            Q[at] *= exp_of(b);
            K[at] *= exp_of(end - b);
        }
        __syncthreads();
        // blocks of earlier tokens: q (block bi) . k (block bj) with the decays of the blocks between
        if (warp < 12) {
            const int pair = warp >> 1, half = warp & 1;
            const int bi = pair == 0 ? 1 : pair < 3 ? 2 : 3, bj = pair == 0 ? 0 : pair < 3 ? pair - 1 : pair - 3;
            float acc[4];
            const float* f0 = bi - bj >= 2 ? Pb + (bj + 1) * RP : nullptr;
            const float* f1 = bi - bj >= 3 ? Pb + (bj + 2) * RP : nullptr;
            token_block<RP>(Q, K, bi * BLOCK, bj * BLOCK + half * 8, f0, f1, gid, tig, acc);
            float* a = A + (bi * BLOCK + gid) * AP + bj * BLOCK + half * 8 + 2 * tig;
            a[0] = acc[0]; a[1] = acc[1]; a[8 * AP] = acc[2]; a[8 * AP + 1] = acc[3];
        }
    } else {
        for (int task = warp; task < 20; task += 16) {       // q k^T of the blocks on and below the diagonal
            const int pair = task >> 1, half = task & 1;
            const int bi = pair < 1 ? 0 : pair < 3 ? 1 : pair < 6 ? 2 : 3, bj = pair - bi * (bi + 1) / 2;
            float acc[4];
            token_block<RP>(Q, K, bi * BLOCK, bj * BLOCK + half * 8, nullptr, nullptr, gid, tig, acc);
            // times the decay from j to i and j's strength, head by head; nothing above the diagonal
            for (int hh = 0; hh < p.hp; ++hh)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = bi * BLOCK + gid + 8 * (e >> 1), j = bj * BLOCK + half * 8 + 2 * tig + (e & 1);
                    A[(hh * CHUNK + i) * AP + j] =
                        j <= i ? acc[e] * wt[hh][j] * exp_of((bc[hh][i] - bc[hh][j]) + (bl[hh][i] - bl[hh][j])) : 0.f;
                }
        }
    }
    cp_async_wait_all();
    __syncthreads();
    // outputs: a warp takes 32 tokens and 16 columns
    const int rp2 = warp & 1, row0 = rp2 * 32, n_base = (warp >> 1) * 16;
    if (n_base >= c.ncols || row0 >= c.nt) return;
    float acc[2][2][4];
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[m][nb][e] = 0.f;
    int hh[2];
    const float* sp[2];                                      // the state's column for this lane's fragment of each block of columns
    int st[2];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
        const int cc = min(n_base + nb * 8 + gid, c.ncols - 1);
        hh[nb] = head_of(p, min(n_base + nb * 8, c.ncols - 1));
        sp[nb] = Ss + cc * P;
        st[nb] = turned(cc);
    }
    const int qt = turned(row0 + gid);                       // rows eight apart are turned alike
#pragma unroll 2
    for (int d0 = 0; d0 < RP; d0 += 16) {
        const int d = d0 + 4 * tig;
        AFrag a0[2], a1[2];
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            const float* qa = Q + (row0 + 16 * m + gid) * P + (d ^ qt);
            float4 x = *reinterpret_cast<const float4*>(qa), y = *reinterpret_cast<const float4*>(qa + 8 * P);
            if (FORM == GATED) {
                const float4 f = *reinterpret_cast<const float4*>(E + (2 * rp2 + m) * RP + d);
                x.x *= f.x; x.y *= f.y; x.z *= f.z; x.w *= f.w;
                y.x *= f.x; y.y *= f.y; y.z *= f.z; y.w *= f.w;
            }
            make_a(a0[m], x.x, y.x, x.y, y.y);
            make_a(a1[m], x.z, y.z, x.w, y.w);
        }
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
            const float4 z = *reinterpret_cast<const float4*>(sp[nb] + (d ^ st[nb]));
            const BFrag b0 = make_b(z.x, z.y), b1 = make_b(z.z, z.w);
            mma_split2(acc[0][nb], acc[1][nb], a0[0], a0[1], b0);
            mma_split2(acc[0][nb], acc[1][nb], a1[0], a1[1], b1);
        }
    }
    if (FORM == HEAD) {
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int nb = 0; nb < 2; ++nb) {
                const float e0 = exp_of(bc[hh[nb]][row0 + 16 * m + gid]), e1 = exp_of(bc[hh[nb]][row0 + 16 * m + gid + 8]);
                acc[m][nb][0] *= e0; acc[m][nb][1] *= e0; acc[m][nb][2] *= e1; acc[m][nb][3] *= e1;
            }
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
        const int i0 = row0 + 16 * m + gid, i1 = i0 + 8, steps = 2 * (2 * rp2 + m + 1);
        for (int ks = 0; ks < steps; ++ks) {
            const int j0 = ks * 8 + tig, j1 = j0 + 4;
            AFrag a;
#pragma unroll
            for (int nb = 0; nb < 2; ++nb) {
                if (nb == 0 || (FORM == HEAD && hh[1] != hh[0])) {
                    const float* Ah = A + (FORM == HEAD ? hh[nb] * CHUNK * AP : 0);
                    make_a(a, Ah[i0 * AP + j0], Ah[i1 * AP + j0], Ah[i0 * AP + j1], Ah[i1 * AP + j1]);
                }
                const float* vb = Vs + j0 * VP + n_base + nb * 8 + gid;
                mma_split(acc[m][nb], a, make_b(vb[0], vb[4 * VP]));
            }
        }
    }
    float* out = p.out + (size_t)c.t0 * p.out_stride + first_column(p, c);
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int cc = n_base + nb * 8 + 2 * tig + e;
            if (cc >= c.ncols) continue;
            const float skip = FORM == HEAD && p.skip ? p.skip[c.h0 + hh[nb]] : 0.f;
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const int i = row0 + 16 * m + gid + 8 * r;
                    if (i < c.nt) out[(size_t)i * p.out_stride + cc] = fmaf(skip, Vs[i * VP + cc], acc[m][nb][e + 2 * r] * p.q_scale);
                }
        }
}

template <int FORM, int RP>
int run(const ChunkParams& p, int n_chunks, int n_seqs, cudaStream_t stream) {
    const size_t s1 = (size_t)(CHUNK * (RP + 8) + CHUNK * VP + (FORM == GATED ? 256 : MAX_HP * CHUNK)) * sizeof(float);
    const size_t s3 = OutputLayout<FORM, RP>::total * sizeof(float);
    static bool sized = false;          // once: the attribute is a property of the function, not of a launch
    if (!sized) {
        cudaFuncSetAttribute(chunk_state_kernel<FORM, RP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        cudaFuncSetAttribute(chunk_output_kernel<FORM, RP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
        sized = true;
    }
    const dim3 grid((unsigned)n_chunks, (unsigned)(p.heads / p.hp * p.col_tiles));
    chunk_state_kernel<FORM, RP><<<grid, 256, s1, stream>>>(p);
    int rc = rs_launch_result();
    if (rc) return rc;
    chunk_scan_kernel<FORM><<<dim3((unsigned)((p.columns * (RP / 4) + 255) / 256), (unsigned)p.heads, (unsigned)n_seqs), 256, 0, stream>>>(p, RP);
    rc = rs_launch_result();
    if (rc) return rc;
    chunk_output_kernel<FORM, RP><<<grid, 512, s3, stream>>>(p);
    return rs_launch_result();
}
}  // namespace

RS_EXPORT int rs_state_chunk_tokens() { return CHUNK; }

// whether the chunked form takes a recurrence of this form, row count (padded) and column count
RS_EXPORT int rs_state_chunks_supported(int form, int rows_pad, int columns) {
    if (rows_pad != 32 && rows_pad != 64 && rows_pad != 128) return 0;
    return form == GATED || (form == HEAD && columns % 8 == 0) ? 1 : 0;
}

// sums: n_chunks * heads * columns * rows_pad floats, decays: n_chunks * heads * rows_pad floats of workspace.  g holds LOG
// decays.  chunk_seq / chunk_start: sequence and first token (within the sequence's portion) of every chunk, the chunks of a
// sequence in order; seq_first_chunk: [n_seqs + 1].
RS_EXPORT int rs_state_recurrence_chunked(const float* q, long q_stride, const float* k, long k_stride, const float* g, long g_stride,
                                          const float* beta, long beta_stride, const float* v, long v_stride, float* out,
                                          long out_stride, float* state, long state_stride, const int* q_start, const int* slots,
                                          const int* chunk_seq, const int* chunk_start, const int* seq_first_chunk, float* sums,
                                          float* decays, int n_chunks, int n_seqs, int heads, int group, int rows, int rows_pad,
                                          int columns, int form, float q_scale, const float* skip, cudaStream_t stream) {
    if (n_chunks <= 0) return 0;
    if (!rs_state_chunks_supported(form, rows_pad, columns) || rows < 4 || rows % 4 || rows > rows_pad || group < 1 || heads % group ||
        (form == HEAD && !beta))
        return (int)cudaErrorInvalidValue;
    const int hp = form == HEAD && group % 2 == 0 && 2 * columns <= COLS ? 2 : 1;       // two heads that share q and k in a CTA
    ChunkParams p{q, q_stride, k, k_stride, g, g_stride, beta, beta_stride, v, v_stride, out, out_stride, state, state_stride, q_start,
                  slots, chunk_seq, chunk_start, seq_first_chunk, sums, decays, heads, group, columns, rows, hp,
                  hp > 1 ? 1 : (columns + COLS - 1) / COLS, q_scale, skip};
#define RS_CHUNKS(F, R) if (form == F && rows_pad == R) return run<F, R>(p, n_chunks, n_seqs, stream);
    RS_CHUNKS(GATED, 32) RS_CHUNKS(GATED, 64) RS_CHUNKS(GATED, 128) RS_CHUNKS(HEAD, 32) RS_CHUNKS(HEAD, 64) RS_CHUNKS(HEAD, 128)
#undef RS_CHUNKS
    return (int)cudaErrorInvalidValue;
}
