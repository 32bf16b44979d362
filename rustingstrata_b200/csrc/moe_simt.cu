// Mixture of experts whose choice is a table from token id to expert ids or a router's, on CUDA cores with float32
// accumulation, for both engines:
//   * router_topk: the choice a router's logits make, a warp per token;
//   * moe_route: the step's (token, k) pairs sorted by expert, entirely on the device: counts, offsets, the list of
//     row tiles (expert, first sorted row, rows) that the grouped products walk;
//   * grouped_linear: one launch for all experts; a CTA takes one row tile of one expert and one tile of output
//     columns, gathers its input rows through the sorted list and writes each pair's result to the pair's own row.
//     Epilogues: plain store, or SiLU(gate) * up with gate rows [0, N) and up rows [N, 2N) of the expert's matrix.
//     A tile of at most 8 rows takes the row-streaming form (a warp per output column, the expert's matrix read
//     once, coalesced); larger tiles the 64 x 64 register-tiled form;
//   * moe_combine: out[t] = sum_k pair_out[t, k] * weight + gate[t] * shared[t], the sum over k in ascending k, so a token's
//     result does not depend on the batch; a pair whose choice is an identity expert contributes h[t]; the whole may be
//     scaled, added to the residual stream, and the stream's new row left in the activation type for its next reader.
// Choices from E on (up to ``identity`` of them) are identity experts: they have no matrices and get no rows in the lists.
// Every pair's row is computed with k ascending whatever else is in the batch.
#include "common.cuh"
#include <math.h>

namespace {
__device__ __forceinline__ void store_any(void* p, int dt, size_t i, float v) {
    if (dt == RS_F32) reinterpret_cast<float*>(p)[i] = v;
    else reinterpret_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16_rn(v);
}
constexpr int MAX_EXPERTS = 4096;
}  // namespace

namespace {
// one warp per token: scores = softmax(logits), or sigmoid(logits) each for itself (``sigmoid``); the `top` largest of
// scores + correction are chosen (the lower index on a tie); with ``n_groups`` > 0 the experts form that many equal
// groups of neighbours, a group is worth the sum of its two largest scores + correction (``worth_one``: its largest), and only experts of the
// ``keep`` groups worth most can be chosen (the lower index on a tie); weights = the chosen experts' scores times
// ``scale``, divided by (their sum + 1e-20) first when ``renorm`` is set
struct RouterParams {
    const float* logits; long l_stride;
    const void* corr; int corr_dt;
    int E, top, n_tokens, sigmoid, n_groups, keep, worth_one;
    float scale;
    int renorm;
    int* choice; float* weight;
    int* status;
};

// The choice of token t by one warp; ``score`` is the warp's shared memory, 2 E + 2 n_groups floats.
__device__ __forceinline__ void router_token(const RouterParams& p, int t, float* score) {
    const float* logits = p.logits; const long l_stride = p.l_stride;
    const void* corr = p.corr; const int corr_dt = p.corr_dt;
    const int E = p.E, top = p.top, n_groups = p.n_groups, keep = p.keep, worth_one = p.worth_one, renorm = p.renorm;
    const float scale = p.scale;
    int* choice = p.choice; float* weight = p.weight; int* status = p.status;
    const bool sigmoid = p.sigmoid != 0;
    const int lane = threadIdx.x & 31;
    float* pick = score + E;
    float* worth = pick + E;                 // [n_groups]
    float* kept = worth + n_groups;          // [n_groups] 1: the group's experts can be chosen
    const float* z = logits + (size_t)t * l_stride;
    if (sigmoid) {
        bool bad = false;
        for (int e = lane; e < E; e += 32) {
            const float v = ld_dep(z + e);
            bad |= !isfinite(v);
            score[e] = 1.0f / (1.0f + expf(-v));
        }
        if (__any_sync(0xffffffffu, bad) && lane == 0) atomicOr(status, RS_STATUS_NON_FINITE);
    } else {
        float m = -INFINITY;
        for (int e = lane; e < E; e += 32) m = fmaxf(m, ld_dep(z + e));
        m = warp_max(m);
        float sum = 0.f;
        for (int e = lane; e < E; e += 32) { const float v = expf(ld_dep(z + e) - m); score[e] = v; sum += v; }
        sum = warp_sum(sum);
        if (!(sum > 0.f) || !isfinite(sum)) { if (lane == 0) atomicOr(status, RS_STATUS_NON_FINITE); }
        for (int e = lane; e < E; e += 32) score[e] = score[e] / sum;
    }
    for (int e = lane; e < E; e += 32) pick[e] = corr != nullptr ? score[e] + load_any(corr, corr_dt, e) : score[e];
    __syncwarp();
    if (n_groups > 0) {
        const int per = E / n_groups;
        for (int g = lane; g < n_groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;              // the group's largest and second largest
            for (int e = g * per; e < (g + 1) * per; ++e) {
                const float v = pick[e];
                if (v > a) { b = a; a = v; } else if (v > b) { b = v; }
            }
            worth[g] = per > 1 && !worth_one ? a + b : a;
            kept[g] = 0.f;
        }
        __syncwarp();
        for (int k = 0; k < keep; ++k) {
            float best = -INFINITY; int bi = 0x7FFFFFFF;
            for (int g = lane; g < n_groups; g += 32) { const float v = worth[g]; if (kept[g] == 0.f && (v > best || bi == 0x7FFFFFFF)) { best = v; bi = g; } }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
                if (oi != 0x7FFFFFFF && (bi == 0x7FFFFFFF || ov > best || (ov == best && oi < bi))) { best = ov; bi = oi; }
            }
            if (bi >= 0 && bi < n_groups && lane == 0) kept[bi] = 1.f;
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32) if (kept[e / per] == 0.f) pick[e] = -INFINITY;
        __syncwarp();
    }
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY; int bi = 0x7FFFFFFF;
        for (int e = lane; e < E; e += 32) { const float v = pick[e]; if (v > best) { best = v; bi = e; } }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
        }
        if (bi < 0 || bi >= E) bi = 0;                           // nothing finite left: every lane agrees
        const float s = score[bi];
        total += s;
        if (lane == 0) { choice[(size_t)t * top + k] = bi; weight[(size_t)t * top + k] = s; pick[bi] = -INFINITY; }
        __syncwarp();
    }
    const float f = renorm ? scale / (total + 1e-20f) : scale;
    __syncwarp();
    for (int k = lane; k < top; k += 32) weight[(size_t)t * top + k] *= f;
}

__global__ void router_topk_kernel(const RouterParams p) {
    extern __shared__ float sm[];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, t = blockIdx.x * (blockDim.x >> 5) + warp;
    if (t < p.n_tokens) router_token(p, t, sm + (size_t)warp * (2 * p.E + 2 * p.n_groups));
}

struct RouteParams {
    const int* ids; const int* table; int V, top, E, identity, n_tokens, rows_per_tile;
    int* order; int* tiles; int* n_tiles; int max_tiles;
    int* status;
};

// order[P]: pair ids (t * top + k) grouped by expert; tiles[i] = (expert, first row in order, rows); n_tiles[0].  By one block;
// counts and cursor hold E numbers each in shared memory.
__device__ __forceinline__ void route_pairs(const RouteParams& p, int* counts, int* cursor) {
    const int P = p.n_tokens * p.top, E = p.E;
    for (int e = threadIdx.x; e < E; e += blockDim.x) counts[e] = 0;
    __syncthreads();
    // the expert of a pair, or -1 for an identity expert's
    auto expert_of = [&](int pr) {
        int id = p.ids != nullptr ? ld_dep(p.ids + pr / p.top) : pr / p.top;       // without ids the table has one row per token of the step
        if (id < 0 || id >= p.V) { atomicOr(p.status, RS_STATUS_BAD_TOKEN); id = 0; }
        const int e = ld_dep(p.table + (size_t)id * p.top + pr % p.top);
        if (e >= E && e < E + p.identity) return -1;
        if (e < 0 || e >= E) { atomicOr(p.status, RS_STATUS_BAD_PLAN); return 0; }
        return e;
    };
    for (int pr = threadIdx.x; pr < P; pr += blockDim.x) {
        const int e = expert_of(pr);
        if (e >= 0) atomicAdd(&counts[e], 1);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int off = 0, nt = 0;
        for (int e = 0; e < E; ++e) {
            cursor[e] = off;
            for (int r0 = 0; r0 < counts[e]; r0 += p.rows_per_tile) {
                if (nt < p.max_tiles) {
                    p.tiles[3 * nt] = e; p.tiles[3 * nt + 1] = off + r0; p.tiles[3 * nt + 2] = min(p.rows_per_tile, counts[e] - r0);
                }
                ++nt;
            }
            off += counts[e];
        }
        if (nt > p.max_tiles) { atomicOr(p.status, RS_STATUS_BAD_PLAN); nt = p.max_tiles; }
        p.n_tiles[0] = nt;
    }
    __syncthreads();
    // Where a pair lands within its expert's rows changes no value: every pair's row is computed by itself.
    for (int pr = threadIdx.x; pr < P; pr += blockDim.x) {
        const int e = expert_of(pr);
        if (e >= 0) p.order[atomicAdd(&cursor[e], 1)] = pr;
    }
}

__global__ void __launch_bounds__(1024) moe_route_kernel(const RouteParams p) {
    __shared__ int counts[MAX_EXPERTS];
    __shared__ int cursor[MAX_EXPERTS];
    pdl_launch_dependents();
    pdl_wait();
    route_pairs(p, counts, cursor);
}

// Choice and lists of a step of few tokens in one block: a warp per token, then the pairs are dealt.
__global__ void __launch_bounds__(1024) router_route_kernel(const RouterParams rp, const RouteParams p) {
    extern __shared__ float sm[];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, warps = blockDim.x >> 5, per = 2 * rp.E + 2 * rp.n_groups;
    if (warp < rp.n_tokens) router_token(rp, warp, sm + (size_t)warp * per);
    __syncthreads();                                   // the choices are in global memory, written by this block
    int* counts = reinterpret_cast<int*>(sm + (size_t)warps * per);
    route_pairs(p, counts, counts + p.E);
}

// Shared memory of the joint form with ``warps`` warps.
size_t router_route_smem(int n_choices, int n_groups, int n_experts, int warps) {
    return ((size_t)warps * (2 * n_choices + 2 * n_groups) + 2 * n_experts) * sizeof(float);
}
}  // namespace

RS_EXPORT int rs_moe_route(const int* ids, const int* table, int V, int top, int E, int identity, int n_tokens, int rows_per_tile,
                           int* order, int* tiles, int* n_tiles, int max_tiles, int* status, void* stream) {
    if (n_tokens <= 0) return 0;
    if (E <= 0 || E > MAX_EXPERTS || identity < 0 || top <= 0 || rows_per_tile <= 0) return (int)cudaErrorInvalidValue;
    const RouteParams p{ids, table, V, top, E, identity, n_tokens, rows_per_tile, order, tiles, n_tiles, max_tiles, status};
    return rs_launch_pdl(moe_route_kernel, dim3(1), dim3(1024), 0, (cudaStream_t)stream, p);
}

RS_EXPORT int rs_router_topk(const float* logits, long l_stride, const void* corr, int corr_dt, int E, int top, int n_tokens,
                             int sigmoid, int n_groups, int keep, int worth_one, float scale, int renorm, int* choice, float* weight,
                             int* status, void* stream) {
    if (n_tokens <= 0) return 0;
    if (E <= 0 || top <= 0 || top > E || E > 1024) return (int)cudaErrorInvalidValue;
    if (n_groups < 0 || (n_groups > 0 && (E % n_groups || keep < 1 || keep > n_groups || top > keep * (E / n_groups))))
        return (int)cudaErrorInvalidValue;
    const RouterParams p{logits, l_stride, corr, corr_dt, E, top, n_tokens, sigmoid, n_groups, keep, worth_one, scale, renorm, choice,
                         weight, status};
    const int wpb = 4;
    return rs_launch_pdl(router_topk_kernel, dim3((n_tokens + wpb - 1) / wpb), dim3(wpb * 32),
                         (size_t)wpb * (2 * E + 2 * n_groups) * sizeof(float), (cudaStream_t)stream, p);
}

// Whether the joint form of the two takes a step of this size.
RS_EXPORT int rs_router_route_supported(int n_tokens, int n_choices, int n_groups, int n_experts) {
    return n_tokens > 0 && n_tokens <= 32 && router_route_smem(n_choices, n_groups, n_experts, n_tokens < 4 ? 4 : n_tokens) <= 48 * 1024;
}

// rs_router_topk over E + identity choices followed by rs_moe_route on what it chose, in one launch.
RS_EXPORT int rs_router_route(const float* logits, long l_stride, const void* corr, int corr_dt, int E, int identity, int top,
                              int n_tokens, int sigmoid, int n_groups, int keep, int worth_one, float scale, int renorm, int* choice,
                              float* weight, int rows_per_tile, int* order, int* tiles, int* n_tiles, int max_tiles, int* status,
                              void* stream) {
    if (n_tokens <= 0) return 0;
    const int n = E + identity;
    if (E <= 0 || identity < 0 || top <= 0 || top > n || n > 1024 || rows_per_tile <= 0 || !rs_router_route_supported(n_tokens, n, n_groups, E))
        return (int)cudaErrorInvalidValue;
    if (n_groups < 0 || (n_groups > 0 && (n % n_groups || keep < 1 || keep > n_groups || top > keep * (n / n_groups))))
        return (int)cudaErrorInvalidValue;
    const RouterParams rp{logits, l_stride, corr, corr_dt, n, top, n_tokens, sigmoid, n_groups, keep, worth_one, scale, renorm, choice,
                          weight, status};
    const RouteParams p{nullptr, choice, n_tokens, top, E, identity, n_tokens, rows_per_tile, order, tiles, n_tiles, max_tiles, status};
    const int warps = n_tokens < 4 ? 4 : n_tokens;              // four warps at least: the lists are dealt by all threads
    return rs_launch_pdl(router_route_kernel, dim3(1), dim3(warps * 32), router_route_smem(n, n_groups, E, warps),
                         (cudaStream_t)stream, rp, p);
}

namespace {
constexpr int GL_BM = 64, GL_BN = 64, GL_BK = 16;

struct GroupedParams {
    const void* a; int a_dt; long a_stride; int a_div;       // input row of a pair = pair / a_div
    const void* w; int w_dt; long w_expert_stride;           // [E][rows][K], rows = N (plain) or 2N (gated)
    void* out; int out_dt; long out_stride;                  // [P, N]
    const int* order; const int* tiles; const int* n_tiles;
    int N, K, gated;          // gated: 0 plain; 1 gate rows [0, N) and up rows [N, 2N); 2 gate row 2n, up row 2n + 1
    int relu2;                // plain products only: out = max(a W.T, 0)^2
};

__device__ __forceinline__ float relu_squared(float v) { v = fmaxf(v, 0.f); return v * v; }

__device__ __forceinline__ size_t gate_row(const GroupedParams& p, int n) { return p.gated == 2 ? 2 * (size_t)n : (size_t)n; }
__device__ __forceinline__ size_t up_row(const GroupedParams& p, int n) { return p.gated == 2 ? 2 * (size_t)n + 1 : (size_t)p.N + n; }

__device__ __forceinline__ float silu_exact(float g) { return g / (1.0f + expf(-g)); }

// 64 x 64 register-tiled form
__global__ void __launch_bounds__(256) grouped_linear_tile_kernel(const GroupedParams p) {
    if ((int)blockIdx.y >= p.n_tiles[0]) return;
    __shared__ float As[GL_BK][GL_BM + 1];
    __shared__ float Ws[GL_BK][GL_BN + 1];
    __shared__ float Us[GL_BK][GL_BN + 1];
    __shared__ int pair_of_row[GL_BM];
    const int e = p.tiles[3 * blockIdx.y], row0 = p.tiles[3 * blockIdx.y + 1], rows = p.tiles[3 * blockIdx.y + 2];
    const int tid = threadIdx.x, n0 = blockIdx.x * GL_BN;
    const int tx = tid % 16, ty = tid / 16;
    if (tid < GL_BM) pair_of_row[tid] = tid < rows ? p.order[row0 + tid] : -1;
    __syncthreads();
    float acc[4][4], accu[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) { acc[i][j] = 0.f; accu[i][j] = 0.f; }
    const size_t wb = (size_t)e * p.w_expert_stride;
    for (int k0 = 0; k0 < p.K; k0 += GL_BK) {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const int idx = tid + q * 256;
            const int r = idx / GL_BK, kk = idx % GL_BK;
            const int gk = k0 + kk, gn = n0 + r;
            const int pr = pair_of_row[r];
            As[kk][r] = (pr >= 0 && gk < p.K) ? load_any(p.a, p.a_dt, (size_t)(pr / p.a_div) * p.a_stride + gk) : 0.f;
            const bool ok = gn < p.N && gk < p.K;
            Ws[kk][r] = ok ? load_any(p.w, p.w_dt, wb + gate_row(p, gn) * p.K + gk) : 0.f;
            if (p.gated) Us[kk][r] = ok ? load_any(p.w, p.w_dt, wb + up_row(p, gn) * p.K + gk) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < GL_BK; ++kk) {
            float a[4], w[4], u[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = As[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) { w[j] = Ws[kk][tx * 4 + j]; u[j] = p.gated ? Us[kk][tx * 4 + j] : 0.f; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
                    if (p.gated) accu[i][j] = fmaf(a[i], u[j], accu[i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int pr = pair_of_row[ty * 4 + i];
        if (pr < 0) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int gn = n0 + tx * 4 + j;
            if (gn >= p.N) continue;
            const float v = p.gated ? silu_exact(acc[i][j]) * accu[i][j] : (p.relu2 ? relu_squared(acc[i][j]) : acc[i][j]);
            store_any(p.out, p.out_dt, (size_t)pr * p.out_stride + gn, v);
        }
    }
}

// row-streaming form for tiles of at most 8 rows: the rows sit in shared memory as float32, a warp owns output
// columns and reads their weight rows once, lanes striding over k.
constexpr int GR_ROWS = 8, GR_COLS = 32, GR_KC = 1024;

__global__ void __launch_bounds__(256) grouped_linear_rows_kernel(const GroupedParams p) {
    if ((int)blockIdx.y >= p.n_tiles[0]) return;
    __shared__ float As[GR_ROWS][GR_KC];
    __shared__ int pair_of_row[GR_ROWS];
    const int e = p.tiles[3 * blockIdx.y], row0 = p.tiles[3 * blockIdx.y + 1], rows = p.tiles[3 * blockIdx.y + 2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int n0 = blockIdx.x * GR_COLS;
    if (tid < GR_ROWS) pair_of_row[tid] = tid < rows ? p.order[row0 + tid] : -1;
    constexpr int CPW = GR_COLS / 8;                          // columns per warp
    float acc[CPW][GR_ROWS], accu[CPW][GR_ROWS];
#pragma unroll
    for (int c = 0; c < CPW; ++c)
#pragma unroll
        for (int r = 0; r < GR_ROWS; ++r) { acc[c][r] = 0.f; accu[c][r] = 0.f; }
    const size_t wb = (size_t)e * p.w_expert_stride;
    const bool vec = p.w_dt == RS_BF16 && p.K % 8 == 0 && p.w_expert_stride % 8 == 0 && ((size_t)p.w & 15) == 0;
    for (int k0 = 0; k0 < p.K; k0 += GR_KC) {
        __syncthreads();
        const int kc = min(GR_KC, p.K - k0);
        for (int i = tid; i < GR_ROWS * kc; i += 256) {
            const int r = i / kc, kk = i % kc;
            const int pr = pair_of_row[r];
            As[r][kk] = pr >= 0 ? load_any(p.a, p.a_dt, (size_t)(pr / p.a_div) * p.a_stride + k0 + kk) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < CPW; ++c) {
            const int gn = n0 + warp * CPW + c;
            if (gn >= p.N) continue;
            const size_t wrow = wb + gate_row(p, gn) * p.K + k0, urow = wb + up_row(p, gn) * p.K + k0;
            if (vec) {
                // eight bfloat16 weights per lane and load (16 bytes), the rows' values from shared memory
                const __nv_bfloat16* wp = reinterpret_cast<const __nv_bfloat16*>(p.w);
                for (int kk = lane * 8; kk < kc; kk += 256) {
                    const uint4 wv = *reinterpret_cast<const uint4*>(wp + wrow + kk);
                    uint4 uv = make_uint4(0, 0, 0, 0);
                    if (p.gated) uv = *reinterpret_cast<const uint4*>(wp + urow + kk);
                    const __nv_bfloat162* w2 = reinterpret_cast<const __nv_bfloat162*>(&wv);
                    const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uv);
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        const float w0 = __low2float(w2[q]), w1 = __high2float(w2[q]);
                        const float u0 = __low2float(u2[q]), u1 = __high2float(u2[q]);
#pragma unroll
                        for (int r = 0; r < GR_ROWS; ++r) {
                            const float a0 = As[r][kk + 2 * q], a1 = As[r][kk + 2 * q + 1];
                            acc[c][r] = fmaf(a1, w1, fmaf(a0, w0, acc[c][r]));
                            if (p.gated) accu[c][r] = fmaf(a1, u1, fmaf(a0, u0, accu[c][r]));
                        }
                    }
                }
                continue;
            }
            for (int kk = lane; kk < kc; kk += 32) {
                const float w = load_any(p.w, p.w_dt, wrow + kk);
                const float u = p.gated ? load_any(p.w, p.w_dt, urow + kk) : 0.f;
#pragma unroll
                for (int r = 0; r < GR_ROWS; ++r) {
                    acc[c][r] = fmaf(As[r][kk], w, acc[c][r]);
                    if (p.gated) accu[c][r] = fmaf(As[r][kk], u, accu[c][r]);
                }
            }
        }
    }
#pragma unroll
    for (int c = 0; c < CPW; ++c) {
        const int gn = n0 + warp * CPW + c;
#pragma unroll
        for (int r = 0; r < GR_ROWS; ++r) {
            const float g = warp_sum(acc[c][r]);
            const float u = p.gated ? warp_sum(accu[c][r]) : 0.f;
            const int pr = pair_of_row[r];
            if (lane == 0 && gn < p.N && pr >= 0)
                store_any(p.out, p.out_dt, (size_t)pr * p.out_stride + gn, p.gated ? silu_exact(g) * u : (p.relu2 ? relu_squared(g) : g));
        }
    }
}
}  // namespace

RS_EXPORT int rs_grouped_linear_rows_per_tile(int small) { return small ? GR_ROWS : GL_BM; }

RS_EXPORT int rs_grouped_linear(const void* a, int a_dt, long a_stride, int a_div, const void* w, int w_dt,
                                long w_expert_stride, void* out, int out_dt, long out_stride, const int* order,
                                const int* tiles, const int* n_tiles, int max_tiles, int N, int K, int gated, int small,
                                int relu2, void* stream) {
    if (max_tiles <= 0 || N <= 0) return 0;
    if (gated && relu2) return (int)cudaErrorInvalidValue;
    GroupedParams p{a, a_dt, a_stride, a_div, w, w_dt, w_expert_stride, out, out_dt, out_stride, order, tiles, n_tiles,
                    N, K, gated, relu2};
    cudaStream_t s = (cudaStream_t)stream;
    if (small) grouped_linear_rows_kernel<<<dim3((N + GR_COLS - 1) / GR_COLS, max_tiles), 256, 0, s>>>(p);
    else grouped_linear_tile_kernel<<<dim3((N + GL_BN - 1) / GL_BN, max_tiles), 256, 0, s>>>(p);
    return rs_launch_result();
}

// y[t, :] = scale * (weight * sum_k (pair_w[t * top + k] or 1) * v_k + g * shared[t, :]), where v_k is pair_out[t * top + k, :],
// or h[t, :] for a pair whose choice is an identity expert (choice[t * top + k] >= n_experts), and g is 1,
// sigmoid(gate_z[t]) or sigmoid(h[t, :] . gate_w) (shared == null: no shared expert).
// out (float32 [T, n]) = y, or += y with ``accumulate``; copy (activation type), when given, takes out's new row as well.
struct CombineParams {
    const float* pair_out; long pair_stride; int top; float weight; const float* pair_w; const int* choice; int n_experts;
    const void* shared; int shared_dt; long shared_stride;
    const void* h; int h_dt; long h_stride;
    const void* gate_w; int gate_dt; const float* gate_z; long gate_z_stride;
    float* out; long out_stride; float scale; int accumulate;
    void* copy; int copy_dt; long copy_stride;
    int n;
};

__device__ __forceinline__ float4 load4_any(const void* p, int dt, size_t i) {       // i a multiple of 4
    if (dt == RS_F32) return ld_dep(reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i));
    const uint2 h = ld_dep(reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p) + i));
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&h.x), b = *reinterpret_cast<const __nv_bfloat162*>(&h.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}

template <int V>      // columns a thread takes at a time: 4 (16-byte aligned rows) or 1
__global__ void __launch_bounds__(256) moe_combine_kernel(const CombineParams p) {
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    float gate = p.shared != nullptr ? 1.0f : 0.f;
    if (p.shared != nullptr && p.gate_z != nullptr) {
        gate = 1.0f / (1.0f + expf(-ld_dep(p.gate_z + (size_t)t * p.gate_z_stride)));
    } else if (p.shared != nullptr && p.gate_w != nullptr) {
        float d = 0.f;
        for (int i = threadIdx.x; i < p.n; i += blockDim.x)
            d = fmaf(ld_dep_any(p.h, p.h_dt, (size_t)t * p.h_stride + i), load_any(p.gate_w, p.gate_dt, i), d);
        d = block_sum(d, scratch);
        gate = 1.0f / (1.0f + expf(-d));
    }
    for (int i = threadIdx.x * V; i < p.n; i += blockDim.x * V) {
        float v[V];
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = 0.f;
        for (int k = 0; k < p.top; ++k) {                    // k ascending
            const size_t pr = (size_t)t * p.top + k;
            const float w = p.pair_w != nullptr ? ld_dep(p.pair_w + pr) : 1.0f;
            const bool identity = p.choice != nullptr && ld_dep(p.choice + pr) >= p.n_experts;
            const void* src = identity ? p.h : (const void*)p.pair_out;
            const int dt = identity ? p.h_dt : (int)RS_F32;
            const size_t at = identity ? (size_t)t * p.h_stride + i : pr * p.pair_stride + i;
            if (V == 4) {
                const float4 u = load4_any(src, dt, at);
                v[0] = fmaf(w, u.x, v[0]); v[1 % V] = fmaf(w, u.y, v[1 % V]); v[2 % V] = fmaf(w, u.z, v[2 % V]); v[3 % V] = fmaf(w, u.w, v[3 % V]);
            } else {
                v[0] = fmaf(w, ld_dep_any(src, dt, at), v[0]);
            }
        }
        float sh[V];
#pragma unroll
        for (int j = 0; j < V; ++j) sh[j] = 0.f;
        if (p.shared != nullptr) {
            if (V == 4) {
                const float4 u = load4_any(p.shared, p.shared_dt, (size_t)t * p.shared_stride + i);
                sh[0] = u.x; sh[1 % V] = u.y; sh[2 % V] = u.z; sh[3 % V] = u.w;
            } else {
                sh[0] = ld_dep_any(p.shared, p.shared_dt, (size_t)t * p.shared_stride + i);
            }
        }
        float* o = p.out + (size_t)t * p.out_stride + i;
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = p.scale * fmaf(gate, sh[j], v[j] * p.weight);
        if (V == 4) {
            float4* o4 = reinterpret_cast<float4*>(o);
            if (p.accumulate) { const float4 x = ld_dep(o4); v[0] += x.x; v[1 % V] += x.y; v[2 % V] += x.z; v[3 % V] += x.w; }
            *o4 = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
        } else {
            if (p.accumulate) v[0] += ld_dep(o);
            o[0] = v[0];
        }
        if (p.copy != nullptr) {
            const size_t at = (size_t)t * p.copy_stride + i;
            if (V == 4 && p.copy_dt == RS_BF16)
                *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p.copy) + at) = pack_bf16x4(v[0], v[1 % V], v[2 % V], v[3 % V]);
            else
#pragma unroll
                for (int j = 0; j < V; ++j) store_any(p.copy, p.copy_dt, at + j, v[j]);
        }
    }
}

RS_EXPORT int rs_moe_combine(const float* pair_out, long pair_stride, int top, float weight, const float* pair_w, const int* choice,
                             int n_experts, const void* shared, int shared_dt, long shared_stride, const void* h, int h_dt,
                             long h_stride, const void* gate_w, int gate_dt, const float* gate_z, long gate_z_stride, float* out,
                             long out_stride, float scale, int accumulate, void* copy, int copy_dt, long copy_stride, int n_tokens,
                             int n, void* stream) {
    if (n_tokens <= 0) return 0;
    if ((choice != nullptr || gate_w != nullptr) && h == nullptr) return (int)cudaErrorInvalidValue;
    CombineParams p{pair_out, pair_stride, top, weight, pair_w, choice, n_experts, shared, shared_dt, shared_stride, h, h_dt, h_stride,
                    gate_w, gate_dt, gate_z, gate_z_stride, out, out_stride, scale, accumulate, copy, copy_dt, copy_stride, n};
    auto ok = [](const void* q, int dt, long stride) { return q == nullptr || ((size_t)q % (dt == RS_F32 ? 16 : 8) == 0 && stride % 4 == 0); };
    const bool vec = n % 4 == 0 && ok(pair_out, RS_F32, pair_stride) && ok(shared, shared_dt, shared_stride) && ok(h, h_dt, h_stride) &&
                     ok(out, RS_F32, out_stride) && ok(copy, copy_dt, copy_stride);
    return rs_launch_pdl(vec ? moe_combine_kernel<4> : moe_combine_kernel<1>, dim3(n_tokens), dim3(256), 0, (cudaStream_t)stream, p);
}
