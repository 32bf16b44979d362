// Softmax attention over a paged bfloat16 key/value cache with float32 queries and float32 softmax weights on the
// warp-level tensor cores, for heads that do not mix: a CTA serves the query heads of ONE key/value head (talking_attention_
// mma.cu keeps all heads in a CTA because their scores meet there).  Windows, kept first keys, blocks of positions, sinks
// and head gates as in talking_attention.cu.
//
// Rows of a CTA's 64-row tile are (query, head of the group) pairs; a warp owns 16 of them.  Queries are scaled, split into
// two bfloat16 terms (x = hi + lo, |lo| <= 2^-9 |x|) and held in registers as matrix fragments; per tile of 64 keys (at
// multiples of 64 counted from the sequence's first key) the scores, the online softmax and the weighted values stay in
// registers: only keys and values pass through shared memory, fetched a tile ahead with cp.async.  The weights are split
// like the queries, so both products carry float32 operands; keys and values are the cache's values exactly.
//
// SINGLE: tiles of one query.  Its heads fill one block of 16 rows, so the four warps take 16 of a tile's 64 keys each and
// their sums meet in shared memory at the end.  Either way a tile's keys may be shared out over several CTAs ("parts"),
// whose sums talking_combine_kernel joins.
#include "paged_attention_mma.cuh"

namespace {
constexpr int KEY_TILE = 64;
constexpr int ROWS = 64;
constexpr int THREADS = 128;
constexpr float LN2 = 0.6931471805599453f;

__host__ __device__ inline int row_pitch(int width) { return width + 8; }        // fragment reads without bank conflicts
size_t smem_bytes(int dk, int dv) {
    const size_t tiles = 2ull * KEY_TILE * (row_pitch(dk) + row_pitch(dv)) * 2;
    const size_t merge = 4ull * 16 * (dv + 2) * 4;                               // SINGLE: the warps' sums, after the last tile
    return 3ull * KEY_TILE * sizeof(long long) + (tiles > merge ? tiles : merge);
}

__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// where every key of tile k0 starts in the cache (row of kv head 0; -1: not a key of this walk)
__device__ __forceinline__ void locate(const MmaParams& p, long long* key_at, int s, int k0, int k_begin, int k_end, int i) {
    const int kpos = k0 + i;
    long long at = -1;
    if ((kpos >= k_begin || kpos < p.keep) && kpos < k_end) {
        const int page = p.block_table[(size_t)s * p.table_stride + kpos / p.page_size];
        if (page < 0 || page >= p.num_pages) atomicOr(p.status, RS_STATUS_BAD_PAGE);
        else at = (long long)page * p.page_stride + (long long)(kpos % p.page_size) * p.hdp;
    }
    key_at[i] = at;
}

// one plane's rows of kv head c into shared memory: two threads a key, 16 bytes a copy; rows without a key are zero
__device__ __forceinline__ void fetch(const MmaParams& p, const long long* key_at, __nv_bfloat16* dst, int width, size_t plane, int c, int tid) {
    const int kk = tid >> 1, pitch = row_pitch(width);
    const long long at = key_at[kk];
    __nv_bfloat16* row = dst + (size_t)kk * pitch;
    const __nv_bfloat16* src = p.cache + (at < 0 ? 0 : at) + plane + (size_t)c * p.page_size * p.hdp;
    for (int d = (tid & 1) * 8; d < width; d += 16) {
        if (at >= 0) cp_async16(smem_addr(row + d), src + d);
        else *reinterpret_cast<uint4*>(row + d) = make_uint4(0u, 0u, 0u, 0u);
    }
}

// DK, DV: blocks of 16 coordinates a head may have; SINGLE: one query per tile
template <int DK, int DV, bool SINGLE>
__global__ void __launch_bounds__(THREADS) grouped_attention_kernel(MmaParams p) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    long long* key_at = reinterpret_cast<long long*>(smem_raw);                  // [3][KEY_TILE]
    const int dk = p.dk, dv = p.dv, r = p.H / p.G, c = blockIdx.y;
    const int kp = row_pitch(dk), vp = row_pitch(dv);
    __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(smem_raw + 3 * KEY_TILE * sizeof(long long));     // [2][KEY_TILE][kp]
    __nv_bfloat16* Vs = Ks + 2 * KEY_TILE * kp;                                  // [2][KEY_TILE][vp]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
    const int* wk = p.work + 5 * (size_t)blockIdx.x;
    const int s = wk[0], q0 = wk[1], part = wk[2], parts = wk[3], row_base = wk[4];
    const int t_first = p.q_start[s] + q0;
    const int q_len = p.q_start[s + 1] - p.q_start[s];
    const int nq = min(p.QT, q_len - q0);
    const int pos0 = p.kv_len[s] - q_len + q0;
    const int k_end = pos0 + nq;
    int k_begin = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;
    if (p.chunk > 0) k_begin = max(k_begin, pos0 / p.chunk * p.chunk);
    // the tiles that hold kept first keys, as far as they lie before the window's, then the window's
    const int kt0 = k_begin / KEY_TILE, kt1 = (k_end + KEY_TILE - 1) / KEY_TILE;
    const int n_keep = min((p.keep + KEY_TILE - 1) / KEY_TILE, kt0), n_walk = n_keep + kt1 - kt0;
    const auto tile_at = [&](int t) { return (t < n_keep ? t : kt0 + t - n_keep) * KEY_TILE; };
    const int per = (n_walk + parts - 1) / parts;
    const int t_begin = part * per, t_end = min(n_walk, t_begin + per);

    // the two rows of this lane: query and head of each, and whether it exists
    int qi[2], head[2];
    bool live[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int row = (SINGLE ? 0 : 16 * warp) + gid + 8 * e;
        qi[e] = row / r;
        live[e] = qi[e] < nq;
        if (!live[e]) qi[e] = 0;
        head[e] = c * r + row % r;
    }
    uint32_t qh[DK][4], ql[DK][4];
#pragma unroll
    for (int ks = 0; ks < DK; ++ks) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {                        // rows gid, gid + 8, then the same eight coordinates on
            const int d = ks * 16 + 2 * tig + (e >> 1) * 8;
            float2 x = make_float2(0.f, 0.f);
            if (d < dk && live[e & 1]) {
                const float* src = p.q + (size_t)(t_first + qi[e & 1]) * p.q_stride + (size_t)head[e & 1] * dk + d;
                x = make_float2(src[0] * (p.scale * LOG2E), src[1] * (p.scale * LOG2E));      // scores come out in powers of two
            }
            split_pair(x.x, x.y, qh[ks][e], ql[ks][e]);
        }
    }
    float m_run[2], l_run[2], O[DV][2][4];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const bool sink = p.sink && live[e];
        m_run[e] = sink ? p.sink[head[e]] * LOG2E : -INFINITY;
        l_run[e] = sink && part == 0 && tig == 0 && (!SINGLE || warp == 0) ? 1.f : 0.f;       // summed over a row's lanes at the end
    }
#pragma unroll
    for (int a = 0; a < DV; ++a)
#pragma unroll
        for (int b = 0; b < 2; ++b)
#pragma unroll
            for (int e = 0; e < 4; ++e) O[a][b][e] = 0.f;

    if (t_begin < t_end) {
        if (tid < KEY_TILE) locate(p, key_at, s, tile_at(t_begin), k_begin, k_end, tid);
        else if (t_begin + 1 < t_end) locate(p, key_at + KEY_TILE, s, tile_at(t_begin + 1), k_begin, k_end, tid - KEY_TILE);
        __syncthreads();
        fetch(p, key_at, Ks, dk, 0, c, tid);
        fetch(p, key_at, Vs, dv, (size_t)p.plane_stride, c, tid);
        cp_async_commit();
    }
    constexpr int NB = SINGLE ? 2 : 8, STEP = SINGLE ? 1 : 2;         // blocks of 8 keys a warp scores; fragments of 16 keys at once
    const int key0 = SINGLE ? 16 * warp : 0;
    for (int t = t_begin; t < t_end; ++t) {
        const int i = t - t_begin, buf = i & 1, k0 = tile_at(t);
        const long long* at = key_at + (i % 3) * KEY_TILE;
        cp_async_wait_all();
        __syncthreads();                                     // tile t has landed, nobody reads the other buffer any more
        if (t + 1 < t_end) {
            const long long* next = key_at + ((i + 1) % 3) * KEY_TILE;
            fetch(p, next, Ks + (buf ^ 1) * KEY_TILE * kp, dk, 0, c, tid);
            fetch(p, next, Vs + (buf ^ 1) * KEY_TILE * vp, dv, (size_t)p.plane_stride, c, tid);
            cp_async_commit();
        }
        if (t + 2 < t_end && tid < KEY_TILE) locate(p, key_at + ((i + 2) % 3) * KEY_TILE, s, tile_at(t + 2), k_begin, k_end, tid);
        // ---- scores
        float S[NB][4];
#pragma unroll
        for (int nb = 0; nb < NB; ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[nb][e] = 0.f;
        const int mi = lane >> 3;
        const uint32_t k_addr = smem_addr(Ks + buf * KEY_TILE * kp) + (uint32_t)((key0 + (mi >> 1) * 8 + (lane & 7)) * kp + (mi & 1) * 8) * 2u;
#pragma unroll
        for (int ks = 0; ks < DK; ++ks) {
            if (ks * 16 >= dk) break;
#pragma unroll
            for (int j = 0; j < NB / 2; j += STEP) {
                uint32_t b[STEP][4];                         // two products of one sum never follow each other directly
#pragma unroll
                for (int u = 0; u < STEP; ++u)
                    ldmatrix_x4(k_addr + (uint32_t)((j + u) * 16 * kp + ks * 16) * 2u, b[u][0], b[u][1], b[u][2], b[u][3]);
#pragma unroll
                for (int u = 0; u < 2 * STEP; ++u) mma16816(S[2 * j + u], qh[ks], b[u >> 1][2 * (u & 1)], b[u >> 1][2 * (u & 1) + 1]);
#pragma unroll
                for (int u = 0; u < 2 * STEP; ++u) mma16816(S[2 * j + u], ql[ks], b[u >> 1][2 * (u & 1)], b[u >> 1][2 * (u & 1) + 1]);
            }
        }
        // ---- what the queries do not see (a tile that every query sees whole needs no look)
        const int last = k0 + KEY_TILE - 1, q_last = k_end - 1;
        const bool whole = last <= pos0 && (last < p.keep || ((p.window <= 0 || k0 > q_last - p.window)
                           && (p.chunk <= 0 || k0 >= q_last / p.chunk * p.chunk)));
        if (!whole) {
#pragma unroll
            for (int nb = 0; nb < NB; ++nb)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int kk = key0 + nb * 8 + 2 * tig + (e & 1);
                    if (!sees(p, pos0 + qi[e >> 1], k0 + kk, at[kk])) S[nb][e] = -INFINITY;
                }
        }
        // ---- online softmax
        float alpha[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float mx = -INFINITY;
#pragma unroll
            for (int nb = 0; nb < NB; ++nb) mx = fmaxf(mx, fmaxf(S[nb][2 * e], S[nb][2 * e + 1]));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float m_new = fmaxf(m_run[e], mx);
            const float base = m_new == -INFINITY ? 0.f : m_new;
            alpha[e] = ex2_approx(m_run[e] - base);          // 2^-inf = 0
            m_run[e] = m_new;
            float sum = 0.f;
#pragma unroll
            for (int nb = 0; nb < NB; ++nb) {
                S[nb][2 * e] = ex2_approx(S[nb][2 * e] - base);
                S[nb][2 * e + 1] = ex2_approx(S[nb][2 * e + 1] - base);
                sum += S[nb][2 * e] + S[nb][2 * e + 1];
            }
            l_run[e] = fmaf(l_run[e], m_new == -INFINITY ? 1.f : alpha[e], sum);
        }
#pragma unroll
        for (int a = 0; a < DV; ++a)
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                O[a][b][0] *= alpha[0]; O[a][b][1] *= alpha[0];
                O[a][b][2] *= alpha[1]; O[a][b][3] *= alpha[1];
            }
        // ---- weighted values
        const uint32_t v_addr = smem_addr(Vs + buf * KEY_TILE * vp)
                              + (uint32_t)((key0 + ((lane >> 3) & 1) * 8 + (lane & 7)) * vp + (lane >> 4) * 8) * 2u;
#pragma unroll
        for (int j = 0; j < NB / 2; ++j) {
            uint32_t ah[4], al[4];
#pragma unroll
            for (int e = 0; e < 4; ++e)                      // rows gid, gid + 8, then the same of the next 8 keys
                split_pair(S[2 * j + (e >> 1)][(e & 1) * 2], S[2 * j + (e >> 1)][(e & 1) * 2 + 1], ah[e], al[e]);
#pragma unroll
            for (int a = 0; a < DV; a += 2) {
                if (a * 16 >= dv) break;
                const bool both = (a + 1) * 16 < dv;
                uint32_t b[2][4];
                ldmatrix_x4_trans(v_addr + (uint32_t)(j * 16 * vp + a * 16) * 2u, b[0][0], b[0][1], b[0][2], b[0][3]);
                if (both) ldmatrix_x4_trans(v_addr + (uint32_t)(j * 16 * vp + a * 16 + 16) * 2u, b[1][0], b[1][1], b[1][2], b[1][3]);
                mma16816(O[a][0], ah, b[0][0], b[0][1]);
                mma16816(O[a][1], ah, b[0][2], b[0][3]);
                if (both) { mma16816(O[a + 1][0], ah, b[1][0], b[1][1]); mma16816(O[a + 1][1], ah, b[1][2], b[1][3]); }
                mma16816(O[a][0], al, b[0][0], b[0][1]);
                mma16816(O[a][1], al, b[0][2], b[0][3]);
                if (both) { mma16816(O[a + 1][0], al, b[1][0], b[1][1]); mma16816(O[a + 1][1], al, b[1][2], b[1][3]); }
            }
        }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 1);
        l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 2);
    }
    if constexpr (SINGLE) {
        // the four warps' sums of the same rows, joined in warp order
        float* merge = reinterpret_cast<float*>(Ks);         // [4][16][dv + 2]
        const int pitch = dv + 2;
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float* row = merge + (warp * 16 + gid + 8 * e) * pitch;
#pragma unroll
            for (int a = 0; a < DV; ++a)
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    const int d = a * 16 + b * 8 + 2 * tig;
                    if (d < dv) { row[d] = O[a][b][2 * e]; row[d + 1] = O[a][b][2 * e + 1]; }
                }
            if (tig == 0) { row[dv] = m_run[e]; row[dv + 1] = l_run[e]; }
        }
        __syncthreads();
        for (int hr = warp; hr < r; hr += 4) {               // a warp per head
            const float* rows = merge + hr * pitch;
            float m = -INFINITY, den = 0.f, w[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) m = fmaxf(m, rows[k * 16 * pitch + dv]);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float mk = rows[k * 16 * pitch + dv];
                w[k] = mk == -INFINITY ? 0.f : ex2_approx(mk - m);
                den = fmaf(w[k], rows[k * 16 * pitch + dv + 1], den);
            }
            const int h = c * r + hr;
            float f = 1.f;
            float* dst = nullptr;
            if (parts == 1) {
                f = den > 0.f ? p.out_scale / den : 0.f;
                if (p.gate) f *= p.gate[(size_t)t_first * p.H + h];
            } else {
                const long prow = (long)row_base + part;
                if (prow >= p.partial_rows) { if (lane == 0) atomicOr(p.status, RS_STATUS_BAD_PLAN); continue; }
                dst = p.partial + ((size_t)prow * p.H + h) * pitch;
                if (lane == 0) { dst[dv] = m * LN2; dst[dv + 1] = den; }
            }
            for (int d = lane; d < dv; d += 32) {
                float y = 0.f;
#pragma unroll
                for (int k = 0; k < 4; ++k) y = fmaf(w[k], rows[k * 16 * pitch + d], y);
                if (dst) dst[d] = y;
                else if (p.out_dt == RS_F32) reinterpret_cast<float*>(p.out)[(size_t)t_first * p.out_stride + (size_t)h * dv + d] = y * f;
                else reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)t_first * p.out_stride + (size_t)h * dv + d] = __float2bfloat16_rn(y * f);
            }
        }
        return;
    } else {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            if (!live[e]) continue;
            float* dst = nullptr;
            float f = 1.f;
            if (parts == 1) {
                f = l_run[e] > 0.f ? p.out_scale / l_run[e] : 0.f;
                if (p.gate) f *= p.gate[(size_t)(t_first + qi[e]) * p.H + head[e]];
            } else {
                const long row = (long)row_base + (long)part * nq + qi[e];
                if (row >= p.partial_rows) { if (tig == 0) atomicOr(p.status, RS_STATUS_BAD_PLAN); continue; }
                dst = p.partial + ((size_t)row * p.H + head[e]) * (dv + 2);
                if (tig == 0) { dst[dv] = m_run[e] * LN2; dst[dv + 1] = l_run[e]; }
            }
            const size_t o = (size_t)(t_first + qi[e]) * p.out_stride + (size_t)head[e] * dv;
#pragma unroll
            for (int a = 0; a < DV; ++a)
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    const int d = a * 16 + b * 8 + 2 * tig;
                    if (d >= dv) continue;
                    const float y0 = O[a][b][2 * e] * f, y1 = O[a][b][2 * e + 1] * f;
                    if (dst) *reinterpret_cast<float2*>(dst + d) = make_float2(y0, y1);
                    else if (p.out_dt == RS_F32) *reinterpret_cast<float2*>(reinterpret_cast<float*>(p.out) + o + d) = make_float2(y0, y1);
                    else *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(p.out) + o + d) = __floats2bfloat162_rn(y0, y1);
                }
        }
    }
}

bool grouped_shape_ok(int H, int G, int dk, int dv) {
    return H >= 1 && G >= 1 && H % G == 0 && dk % 16 == 0 && dv % 16 == 0 && dk >= 16 && dv >= 16 && dk <= 128 && dv <= 128 && H / G <= ROWS;
}

template <int DK, int DV, bool SINGLE>
int launch_grouped(const MmaParams& p, int n_work, cudaStream_t stream) {
    const size_t smem = smem_bytes(p.dk, p.dv);
    static size_t sized = 0;            // the most shared memory asked for so far
    if (smem > sized) {
        const cudaError_t e = cudaFuncSetAttribute(grouped_attention_kernel<DK, DV, SINGLE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        sized = smem;
    }
    grouped_attention_kernel<DK, DV, SINGLE><<<dim3((unsigned)n_work, (unsigned)p.G), THREADS, smem, stream>>>(p);
    return rs_launch_result();
}
template <bool SINGLE>
int launch_sizes(const MmaParams& p, int n_work, cudaStream_t stream) {
    if (p.dk <= 64) return p.dv <= 64 ? launch_grouped<4, 4, SINGLE>(p, n_work, stream) : launch_grouped<4, 8, SINGLE>(p, n_work, stream);
    return p.dv <= 64 ? launch_grouped<8, 4, SINGLE>(p, n_work, stream) : launch_grouped<8, 8, SINGLE>(p, n_work, stream);
}
}  // namespace

// queries a tile of the kernel for several queries takes (0: the shape is not one of its shapes)
RS_EXPORT int rs_grouped_attention_q_per_cta(int H, int G, int dk, int dv) {
    return grouped_shape_ok(H, G, dk, dv) ? ROWS / (H / G) : 0;
}
// whether the kernel for single queries takes these head counts
RS_EXPORT int rs_grouped_attention_single_ok(int H, int G, int dk, int dv) {
    return grouped_shape_ok(H, G, dk, dv) && H / G <= 16 ? 1 : 0;
}

// work: n_work rows of (sequence, first query, part, parts, first row of the tile's partial sums) for tiles of QT queries;
// single != 0: tiles of one query (QT 1).  any_parts: some row has parts > 1 (the combine kernel runs).
RS_EXPORT int rs_grouped_attention_mma(const float* q, long q_stride, const float* gate, const void* cache, long page_stride,
                                       int num_pages, int page_size, int hdp, const int* block_table, int table_stride,
                                       const int* q_start, const int* kv_len, const int* work, int n_work, int any_parts,
                                       int single, const float* sink, void* out, int out_dt, long out_stride, float* partial,
                                       long partial_rows, int H, int G, int dk, int dv, int window, int chunk, int keep, int QT,
                                       float scale, float out_scale, int* status, cudaStream_t stream) {
    if (n_work <= 0) return 0;
    if (!grouped_shape_ok(H, G, dk, dv) || hdp % 8 || QT < 1 || (any_parts && !partial) ||
        (single ? QT != 1 || H / G > 16 : QT * (H / G) > ROWS))
        return (int)cudaErrorInvalidValue;
    MmaParams p{q, q_stride, gate, reinterpret_cast<const __nv_bfloat16*>(cache), page_stride, (long)G * page_size * hdp, num_pages,
                page_size, hdp, block_table, table_stride, q_start, kv_len, work, nullptr, sink, out, out_dt, out_stride, partial,
                partial_rows, H, G, dk, dv, window, chunk, keep, QT, scale, out_scale, status};
    const int rc = single ? launch_sizes<true>(p, n_work, stream) : launch_sizes<false>(p, n_work, stream);
    if (rc || !any_parts) return rc;
    talking_combine_kernel<<<n_work, QT * H >= 64 ? 1024 : 256, 0, stream>>>(p);
    return rs_launch_result();
}
