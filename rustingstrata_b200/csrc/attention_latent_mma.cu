// Attention over a one-plane paged cache whose rows are key and value at once (a latent shared by all query heads),
// on the warp-level tensor cores (mma.sync m16n8k16, bfloat16 operands, float32 accumulation), for prompt portions and
// for single query tokens (split form).  The bfloat16 engine's kernel of latent attention for rows of up to 576
// values (a 512-wide latent with a 64-wide rotated part).
//
// Two kernels share the arithmetic.  The narrow one serves single query tokens and short portions, the wide one (64 query
// rows a CTA, at the end of this comment) portions that fill the device with tiles of that size.
//
// Narrow: a CTA of 8 warps owns 16 query rows: (tokens of a tile) x (query heads of a chunk), all reading the same key rows.
// Key tiles of 64 keys are streamed through two shared-memory buffers with cp.async (tile i + 1 loads under tile i), or
// through one where two would keep a second CTA off the SM.
// Per tile:
//   1. S = Q K^T: warp w computes the 16 x 8 block of keys 8w .. 8w + 7 over the whole row width, scales and masks it
//      (causal, window, the split's range) and leaves it in shared memory;
//   2. online softmax in float32: 16 threads per row take the tile's maximum, the probabilities (rounded to bfloat16
//      for the product; with split_p in two bfloat16 terms, p = hi + lo with |lo| <= 2^-9 p, both of which are multiplied,
//      so that the product carries the float32 weight), the running sum and the factor by which the row's earlier
//      results shrink;
//   3. O += P V with V the same key rows: warp w owns a slice of the row's coordinates (an eighth, rounded up to 8).
// Key tiles start at multiples of 64 from key 0 and the split form's splits at multiples of the split size, so the order
// in which a query's keys are reduced depends on its position alone.  The split form leaves un-normalised partial
// results (sum, maximum, denominator) per (sequence, split, head) that a second kernel merges in ascending order,
// the layout and order of the CUDA-core kernel (attention_simt.cu).  With a sink (one learned number per head) the softmax's
// denominator also holds exp(sink): it joins once, where a row's sums are complete.
//
// Wide: a CTA of 12 warps owns 64 query rows and walks key tiles of 48 keys in two buffers, so a key row fetched into shared
// memory serves four times the rows.  S: warp (g, c) computes 16 rows x 16 keys; softmax: four threads a row; O: warp (g, c)
// owns 16 rows and a third of the value columns.  Only the columns that the value map reads (v_cols) are summed.
#include "mma_helpers.cuh"
#include <math.h>
#include <atomic>

namespace {
constexpr int KT = 64, ROWS = 16, WARPS = 8, THREADS = WARPS * 32, NT_MAX = 9, MAX_LAT = 576;
constexpr int S_PITCH = KT + 4, P_PITCH = KT + 8, MERGE_CACHED = 512;

struct LatParams {
    const __nv_bfloat16* q; long q_stride;          // [tokens, q_stride], head h at h * lat
    __nv_bfloat16* out; long out_stride;
    const __nv_bfloat16* cache; long page_stride;   // [pages][page_size][lat]
    int num_pages, page_size;
    const int* block_table; int table_stride;
    const int* q_start; const int* kv_len; const int* work;
    int n_heads, lat, hc, tok_per_cta, window;
    float scale;
    int decode, split_keys, max_splits;
    const int* split_start; float* partial; int partial_slots;
    int* status;
    int n_buf;                                      // key buffers in shared memory: 2 (tile i + 1 loads under tile i) or 1
    int split_p;                                    // 1: the softmax weights enter P V in two bfloat16 terms
    const float* sink;                              // [n_heads] or null: exp(sink[h]) joins the softmax's denominator
    int v_cols;                                     // columns of a row that are summed (a multiple of 8, up to lat)
};

__device__ __forceinline__ void ldmatrix_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}

// KS: k steps of 16 whose query fragments a warp keeps in registers across all key tiles (rows of up to 16 KS values);
// 0: the fragments are read from shared memory at every use (any row width).
template <int KS>
__global__ void __launch_bounds__(THREADS, 1) latent_attention_kernel(const LatParams p) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int lat = p.lat, pitch = lat + 8, chunks = lat >> 3;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);                  // [ROWS][pitch]
    __nv_bfloat16* Ks = Qs + ROWS * pitch;                                          // [n_buf][KT][pitch]
    float* Ss = reinterpret_cast<float*>(Ks + p.n_buf * KT * pitch);                      // [ROWS][S_PITCH]
    __nv_bfloat16* Ps = reinterpret_cast<__nv_bfloat16*>(Ss + ROWS * S_PITCH);      // [ROWS][P_PITCH]
    __nv_bfloat16* Pl = Ps + ROWS * P_PITCH;                                        // [ROWS][P_PITCH] the weights' second terms
    float* stat_m = reinterpret_cast<float*>(Pl + ROWS * P_PITCH);                  // [ROWS] each
    float* stat_l = stat_m + ROWS;
    float* stat_c = stat_l + ROWS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    pdl_launch_dependents();
    pdl_wait();

    int seq, q_off, n_q_tok;
    if (p.decode) { seq = p.work[blockIdx.x]; q_off = 0; n_q_tok = 1; }
    else { seq = p.work[2 * blockIdx.x]; q_off = p.work[2 * blockIdx.x + 1]; }
    const int row0 = p.q_start[seq];
    const int q_len = p.q_start[seq + 1] - row0;
    const int kv_len = p.kv_len[seq];
    if (!p.decode) n_q_tok = min(p.tok_per_cta, q_len - q_off);
    const int qpos0 = kv_len - q_len + q_off;
    const int head0 = blockIdx.y * p.hc;

    int key_lo = p.window > 0 ? max(0, qpos0 - p.window + 1) : 0;
    int key_hi = min(kv_len, qpos0 + n_q_tok);
    int split_local = 0;
    if (p.decode) {
        const int first_split = key_lo / p.split_keys;
        split_local = blockIdx.z;
        const int s = first_split + split_local;
        key_lo = max(key_lo, s * p.split_keys);
        key_hi = min(key_hi, (s + 1) * p.split_keys);
        if (key_lo >= key_hi) return;
    }

    // queries: row r = token (r / hc), head head0 + r % hc; rows beyond the tile's tokens or the model's heads are zero
    for (int i = tid; i < ROWS * chunks; i += THREADS) {
        const int r = i / chunks, ch = i - r * chunks;
        const int tl = r / p.hc, h = head0 + r % p.hc;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (tl < n_q_tok && h < p.n_heads)
            v = ld_dep(reinterpret_cast<const uint4*>(p.q + (size_t)(row0 + q_off + tl) * p.q_stride + (size_t)h * lat + ch * 8));
        *reinterpret_cast<uint4*>(Qs + r * pitch + ch * 8) = v;
    }
    if (tid < ROWS) { stat_m[tid] = -INFINITY; stat_l[tid] = 0.f; stat_c[tid] = 1.f; }

    const int* table = p.block_table + (size_t)seq * p.table_stride;
    auto load_tile = [&](int buf, int k0) {
        __nv_bfloat16* dst0 = Ks + (size_t)buf * KT * pitch;
        for (int i = tid; i < KT * chunks; i += THREADS) {
            const int j = i / chunks, ch = i - j * chunks;
            const int kpos = k0 + j;
            __nv_bfloat16* dst = dst0 + j * pitch + ch * 8;
            bool loaded = false;
            if (kpos >= key_lo && kpos < key_hi) {
                const int page = table[kpos / p.page_size];
                if (page >= 0 && page < p.num_pages) {
                    cp_async16(smem_addr(dst), p.cache + (size_t)page * p.page_stride + (size_t)(kpos % p.page_size) * lat + ch * 8);
                    loaded = true;
                } else if (ch == 0) {
                    atomicOr(p.status, RS_STATUS_BAD_PAGE);
                }
            }
            if (!loaded) *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
    };

    // the slice of the row's coordinates this warp accumulates in step 3
    const int DW = ((p.v_cols + 63) >> 6) << 3;
    const int dim_lo = warp * DW;
    const int my_nt = max(0, min(DW, p.v_cols - dim_lo)) >> 3;
    float acc[NT_MAX][4];
#pragma unroll
    for (int n = 0; n < NT_MAX; ++n) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }

    const int k_first = (key_lo / KT) * KT;
    const int n_tiles = (key_hi - k_first + KT - 1) / KT;
    load_tile(0, k_first);
    cp_async_commit();
    const int a_row = (lane & 7) + 8 * ((lane >> 3) & 1), a_col = 8 * (lane >> 4);
    uint32_t qf[KS > 0 ? KS : 1][4];
    if (KS > 0) {
        __syncthreads();                                       // the queries are in shared memory
        const uint32_t qa = smem_addr(Qs + a_row * pitch + a_col);
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            if (ks * 16 < lat) ldmatrix_x4(qa + ks * 32, qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
            else qf[ks][0] = qf[ks][1] = qf[ks][2] = qf[ks][3] = 0u;
        }
    }
    for (int it = 0; it < n_tiles; ++it) {
        const int k0 = k_first + it * KT;
        if (p.n_buf == 2 && it + 1 < n_tiles) {
            load_tile((it + 1) & 1, k0 + KT);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            if (p.n_buf == 1 && it > 0) {                      // one buffer: the tile is fetched when the last one is done with
                load_tile(0, k0);
                cp_async_commit();
            }
            cp_async_wait<0>();
        }
        __syncthreads();
        const __nv_bfloat16* Kt = Ks + (size_t)(p.n_buf == 2 ? (it & 1) : 0) * KT * pitch;
        // ---- 1. S = Q K^T for this warp's 8 keys
        {
            float c[4] = {0.f, 0.f, 0.f, 0.f};
            const uint32_t qa = smem_addr(Qs + a_row * pitch + a_col);
            const uint32_t kb = smem_addr(Kt + (warp * 8 + (lane & 7)) * pitch + 8 * ((lane >> 3) & 1));
            if (KS > 0) {
#pragma unroll
                for (int ks = 0; ks < KS; ++ks) {
                    if (ks * 16 < lat) {
                        uint32_t b0, b1;
                        ldmatrix_x2(kb + ks * 32, b0, b1);
                        mma16816(c, qf[ks], b0, b1);
                    }
                }
            } else {
                for (int kk = 0; kk < lat; kk += 16) {
                    uint32_t a[4], b0, b1;
                    ldmatrix_x4(qa + kk * 2, a[0], a[1], a[2], a[3]);
                    ldmatrix_x2(kb + kk * 2, b0, b1);
                    mma16816(c, a, b0, b1);
                }
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = (lane >> 2) + 8 * (e >> 1), cc = warp * 8 + (lane & 3) * 2 + (e & 1);
                const int kpos = k0 + cc, qpos = qpos0 + r / p.hc;
                const bool ok = kpos >= key_lo && kpos < key_hi && kpos <= qpos && (p.window <= 0 || kpos > qpos - p.window);
                Ss[r * S_PITCH + cc] = ok ? c[e] * p.scale : -INFINITY;
            }
        }
        __syncthreads();
        // ---- 2. online softmax: 16 threads per row, 4 keys each
        {
            const int r = tid >> 4, j = tid & 15;
            const float4 s4 = *reinterpret_cast<const float4*>(Ss + r * S_PITCH + j * 4);
            float mx = fmaxf(fmaxf(s4.x, s4.y), fmaxf(s4.z, s4.w));
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_old = stat_m[r];
            const float m_new = fmaxf(m_old, mx);
            float p0 = 0.f, p1 = 0.f, p2 = 0.f, p3 = 0.f, corr = 1.f;
            if (m_new != -INFINITY) {
                p0 = __expf(s4.x - m_new); p1 = __expf(s4.y - m_new); p2 = __expf(s4.z - m_new); p3 = __expf(s4.w - m_new);
                corr = __expf(m_old - m_new);
            }
            float sum = (p0 + p1) + (p2 + p3);
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            uint2 pk;
            pk.x = pack_bf16(p0, p1); pk.y = pack_bf16(p2, p3);
            *reinterpret_cast<uint2*>(Ps + r * P_PITCH + j * 4) = pk;
            if (p.split_p) {
                const __nv_bfloat162 h01 = *reinterpret_cast<const __nv_bfloat162*>(&pk.x);
                const __nv_bfloat162 h23 = *reinterpret_cast<const __nv_bfloat162*>(&pk.y);
                uint2 lo;
                lo.x = pack_bf16(p0 - __low2float(h01), p1 - __high2float(h01));
                lo.y = pack_bf16(p2 - __low2float(h23), p3 - __high2float(h23));
                *reinterpret_cast<uint2*>(Pl + r * P_PITCH + j * 4) = lo;
            }
            if (j == 0) { stat_m[r] = m_new; stat_l[r] = stat_l[r] * corr + sum; stat_c[r] = corr; }
        }
        __syncthreads();
        // ---- 3. O = O * corr + P V over this warp's coordinates
        if (my_nt > 0) {
            const float c0 = stat_c[lane >> 2], c1 = stat_c[(lane >> 2) + 8];
#pragma unroll
            for (int n = 0; n < NT_MAX; ++n) { acc[n][0] *= c0; acc[n][1] *= c0; acc[n][2] *= c1; acc[n][3] *= c1; }
            const uint32_t pa = smem_addr(Ps + a_row * P_PITCH + a_col);
            const uint32_t pl = smem_addr(Pl + a_row * P_PITCH + a_col);
            const uint32_t vb = smem_addr(Kt + (lane & 15) * pitch + dim_lo);
#pragma unroll
            for (int kk = 0; kk < KT; kk += 16) {
                uint32_t a[4], al[4] = {0u, 0u, 0u, 0u};
                ldmatrix_x4(pa + kk * 2, a[0], a[1], a[2], a[3]);
                if (p.split_p) ldmatrix_x4(pl + kk * 2, al[0], al[1], al[2], al[3]);
#pragma unroll
                for (int n = 0; n < NT_MAX; ++n) {
                    if (n < my_nt) {
                        uint32_t b0, b1;
                        ldmatrix_x2_trans(vb + (kk * pitch + n * 8) * 2, b0, b1);
                        mma16816(acc[n], a, b0, b1);
                        if (p.split_p) mma16816(acc[n], al, b0, b1);
                    }
                }
            }
        }
        __syncthreads();
    }

    // ---- results: row r = lane / 4 (+ 8), coordinates dim_lo + n * 8 + (lane % 4) * 2 (+ 1)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = (lane >> 2) + 8 * half;
        const int tl = r / p.hc, h = head0 + r % p.hc;
        if (tl >= n_q_tok || h >= p.n_heads) continue;
        if (p.decode) {
            const size_t slot = (size_t)p.split_start[blockIdx.x] + split_local;
            if (slot >= (size_t)p.partial_slots) {
                if ((lane & 3) == 0 && warp == 0) atomicOr(p.status, RS_STATUS_BAD_PLAN);
                continue;
            }
            float* dst = p.partial + (slot * p.n_heads + h) * (lat + 2);
#pragma unroll
            for (int n = 0; n < NT_MAX; ++n) {
                if (n < my_nt) {
                    const int d = dim_lo + n * 8 + (lane & 3) * 2;
                    *reinterpret_cast<float2*>(dst + d) = make_float2(acc[n][2 * half], acc[n][2 * half + 1]);
                }
            }
            if (warp == 0 && (lane & 3) == 0) { dst[lat] = stat_m[r]; dst[lat + 1] = stat_l[r]; }
        } else {
            float inv = 1.0f / stat_l[r];
            if (p.sink != nullptr) {
                const float sk = p.sink[h], M = fmaxf(stat_m[r], sk), e = __expf(stat_m[r] - M);
                inv = e / fmaf(stat_l[r], e, __expf(sk - M));
            }
            __nv_bfloat16* dst = p.out + (size_t)(row0 + q_off + tl) * p.out_stride + (size_t)h * lat;
#pragma unroll
            for (int n = 0; n < NT_MAX; ++n) {
                if (n < my_nt) {
                    const int d = dim_lo + n * 8 + (lane & 3) * 2;
                    *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(acc[n][2 * half] * inv, acc[n][2 * half + 1] * inv);
                }
            }
        }
    }
}

constexpr int WR = 64, WK = 48, WWARPS = 12, WTHREADS = WWARPS * 32, WS_PITCH = WK + 4, WP_PITCH = WK + 8;

__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}

// NT: tiles of 8 value columns a warp accumulates at most (a third of v_cols, rounded up to an even number of tiles).
template <int NT>
__global__ void __launch_bounds__(WTHREADS, 1) latent_portion_kernel(const LatParams p) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int lat = p.lat, pitch = lat + 8, chunks = lat >> 3;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);                  // [WR][pitch]
    __nv_bfloat16* Ks = Qs + WR * pitch;                                            // [2][WK][pitch]
    float* Ss = reinterpret_cast<float*>(Ks + 2 * WK * pitch);                      // [WR][WS_PITCH]
    __nv_bfloat16* Ps = reinterpret_cast<__nv_bfloat16*>(Ss + WR * WS_PITCH);       // [WR][WP_PITCH]
    __nv_bfloat16* Pl = Ps + WR * WP_PITCH;                                         // [WR][WP_PITCH] the weights' second terms
    float* stat_m = reinterpret_cast<float*>(Pl + WR * WP_PITCH);                   // [WR] each
    float* stat_l = stat_m + WR;
    float* stat_c = stat_l + WR;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;

    const int seq = p.work[2 * blockIdx.x], q_off = p.work[2 * blockIdx.x + 1];
    const int row0 = p.q_start[seq];
    const int q_len = p.q_start[seq + 1] - row0;
    const int kv_len = p.kv_len[seq];
    const int n_q_tok = min(p.tok_per_cta, q_len - q_off);
    const int qpos0 = kv_len - q_len + q_off;
    const int head0 = blockIdx.y * p.hc;
    const int n_rows = n_q_tok * p.hc;
    const int key_lo = p.window > 0 ? max(0, qpos0 - p.window + 1) : 0;
    const int key_hi = min(kv_len, qpos0 + n_q_tok);

    for (int i = tid; i < WR * chunks; i += WTHREADS) {        // row r = token (r / hc), head head0 + r % hc
        const int r = i / chunks, ch = i - r * chunks;
        const int tl = r / p.hc, h = head0 + r - tl * p.hc;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < n_rows && h < p.n_heads)
            v = ld_dep(reinterpret_cast<const uint4*>(p.q + (size_t)(row0 + q_off + tl) * p.q_stride + (size_t)h * lat + ch * 8));
        *reinterpret_cast<uint4*>(Qs + r * pitch + ch * 8) = v;
    }
    if (tid < WR) { stat_m[tid] = -INFINITY; stat_l[tid] = 0.f; stat_c[tid] = 1.f; }

    const int* table = p.block_table + (size_t)seq * p.table_stride;
    auto load_tile = [&](int buf, int k0) {                    // eight threads a key row, 16 bytes each in turn
        const int j = tid >> 3, kpos = k0 + j;
        __nv_bfloat16* dst = Ks + ((size_t)buf * WK + j) * pitch;
        const __nv_bfloat16* src = nullptr;
        if (kpos >= key_lo && kpos < key_hi) {
            const int page = table[kpos / p.page_size];
            if (page >= 0 && page < p.num_pages) src = p.cache + (size_t)page * p.page_stride + (size_t)(kpos % p.page_size) * lat;
            else if ((tid & 7) == 0) atomicOr(p.status, RS_STATUS_BAD_PAGE);
        }
        for (int ch = tid & 7; ch < chunks; ch += 8) {
            if (src != nullptr) cp_async16(smem_addr(dst + ch * 8), src + ch * 8);
            else *reinterpret_cast<uint4*>(dst + ch * 8) = make_uint4(0, 0, 0, 0);
        }
    };

    const int rg = (warp & 3) * 16, cg = warp >> 2;            // this warp's row group; its keys (S) and value columns (O)
    const int tiles_v = p.v_cols >> 3, per = ((tiles_v + 2) / 3 + 1) & ~1;
    const int nt_lo = cg * per, my_nt = max(0, min(per, tiles_v - nt_lo));
    float acc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }

    const int k_first = (key_lo / WK) * WK;
    const int n_tiles = (key_hi - k_first + WK - 1) / WK;
    load_tile(0, k_first);
    cp_async_commit();
    const int a_row = (lane & 7) + 8 * ((lane >> 3) & 1), a_col = 8 * (lane >> 4);
    const int b_row = (lane & 7) + 8 * (lane >> 4), b_col = 8 * ((lane >> 3) & 1);
    const uint32_t qa = smem_addr(Qs + (rg + a_row) * pitch + a_col);
    const uint32_t pa = smem_addr(Ps + (rg + a_row) * WP_PITCH + a_col), pl = smem_addr(Pl + (rg + a_row) * WP_PITCH + a_col);
    for (int it = 0; it < n_tiles; ++it) {
        const int k0 = k_first + it * WK;
        cp_async_wait<0>();
        __syncthreads();                                       // the tile is here, and nobody reads the other buffer any more
        if (it + 1 < n_tiles) {
            load_tile((it + 1) & 1, k0 + WK);
            cp_async_commit();
        }
        const __nv_bfloat16* Kt = Ks + (size_t)(it & 1) * WK * pitch;
        // ---- S = Q K^T: 16 rows x 16 keys
        {
            float c[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
            const uint32_t kb = smem_addr(Kt + (cg * 16 + b_row) * pitch + b_col);
#pragma unroll 4
            for (int kk = 0; kk < lat; kk += 16) {
                uint32_t a[4], b[4];
                ldmatrix_x4(qa + kk * 2, a[0], a[1], a[2], a[3]);
                ldmatrix_x4(kb + kk * 2, b[0], b[1], b[2], b[3]);
                mma16816(c[0], a, b[0], b[1]);
                mma16816(c[1], a, b[2], b[3]);
            }
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int r = rg + (lane >> 2) + 8 * half, qpos = qpos0 + r / p.hc;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int cc = cg * 16 + j * 8 + (lane & 3) * 2;
                    float2 s;
                    float* sp = &s.x;
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int kpos = k0 + cc + e;
                        const bool ok = kpos >= key_lo && kpos < key_hi && kpos <= qpos && (p.window <= 0 || kpos > qpos - p.window);
                        sp[e] = ok ? c[j][2 * half + e] * p.scale : -INFINITY;
                    }
                    *reinterpret_cast<float2*>(Ss + r * WS_PITCH + cc) = s;
                }
            }
        }
        __syncthreads();
        // ---- online softmax: four threads a row, 12 keys each
        if (tid < WR * 4) {
            const int r = tid >> 2, j = tid & 3;
            float s[12];
#pragma unroll
            for (int u = 0; u < 3; ++u) {
                const float4 v = *reinterpret_cast<const float4*>(Ss + r * WS_PITCH + j * 12 + u * 4);
                s[4 * u] = v.x; s[4 * u + 1] = v.y; s[4 * u + 2] = v.z; s[4 * u + 3] = v.w;
            }
            float mx = s[0];
#pragma unroll
            for (int u = 1; u < 12; ++u) mx = fmaxf(mx, s[u]);
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float m_old = stat_m[r], m_new = fmaxf(m_old, mx);
            const bool any = m_new != -INFINITY;
            const float corr = any ? __expf(m_old - m_new) : 1.f;
            float sum = 0.f;
#pragma unroll
            for (int u = 0; u < 12; ++u) { s[u] = any ? __expf(s[u] - m_new) : 0.f; sum += s[u]; }
            sum += __shfl_xor_sync(0xffffffffu, sum, 1);
            sum += __shfl_xor_sync(0xffffffffu, sum, 2);
#pragma unroll
            for (int u = 0; u < 3; ++u) {
                uint2 hi, lo;
                hi.x = pack_bf16(s[4 * u], s[4 * u + 1]); hi.y = pack_bf16(s[4 * u + 2], s[4 * u + 3]);
                *reinterpret_cast<uint2*>(Ps + r * WP_PITCH + j * 12 + u * 4) = hi;
                if (p.split_p) {
                    const __nv_bfloat162 h01 = *reinterpret_cast<const __nv_bfloat162*>(&hi.x);
                    const __nv_bfloat162 h23 = *reinterpret_cast<const __nv_bfloat162*>(&hi.y);
                    lo.x = pack_bf16(s[4 * u] - __low2float(h01), s[4 * u + 1] - __high2float(h01));
                    lo.y = pack_bf16(s[4 * u + 2] - __low2float(h23), s[4 * u + 3] - __high2float(h23));
                    *reinterpret_cast<uint2*>(Pl + r * WP_PITCH + j * 12 + u * 4) = lo;
                }
            }
            if (j == 0) { stat_m[r] = m_new; stat_l[r] = stat_l[r] * corr + sum; stat_c[r] = corr; }
        }
        __syncthreads();
        // ---- O = O * corr + P V: 16 rows x this warp's columns
        const float c0 = stat_c[rg + (lane >> 2)], c1 = stat_c[rg + (lane >> 2) + 8];
        if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
            for (int n = 0; n < NT; ++n) { acc[n][0] *= c0; acc[n][1] *= c0; acc[n][2] *= c1; acc[n][3] *= c1; }
        }
        const uint32_t vb = smem_addr(Kt + ((lane & 7) + 8 * ((lane >> 3) & 1)) * pitch + nt_lo * 8 + 8 * (lane >> 4));
#pragma unroll
        for (int kk = 0; kk < WK; kk += 16) {
            uint32_t a[4], al[4] = {0u, 0u, 0u, 0u};
            ldmatrix_x4(pa + kk * 2, a[0], a[1], a[2], a[3]);
            if (p.split_p) ldmatrix_x4(pl + kk * 2, al[0], al[1], al[2], al[3]);
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                if (n < my_nt) {                               // an odd last tile brings the row's padding along: it is not stored
                    uint32_t b[4];
                    ldmatrix_x4_trans(vb + (kk * pitch + n * 8) * 2, b[0], b[1], b[2], b[3]);
                    mma16816(acc[n], a, b[0], b[1]);
                    mma16816(acc[n + 1], a, b[2], b[3]);
                    if (p.split_p) {
                        mma16816(acc[n], al, b[0], b[1]);
                        mma16816(acc[n + 1], al, b[2], b[3]);
                    }
                }
            }
        }
    }

#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = rg + (lane >> 2) + 8 * half;
        const int tl = r / p.hc, h = head0 + r - tl * p.hc;
        if (r >= n_rows || h >= p.n_heads) continue;
        float inv = 1.0f / stat_l[r];
        if (p.sink != nullptr) {
            const float sk = p.sink[h], M = fmaxf(stat_m[r], sk), e = __expf(stat_m[r] - M);
            inv = e / fmaf(stat_l[r], e, __expf(sk - M));
        }
        __nv_bfloat16* dst = p.out + (size_t)(row0 + q_off + tl) * p.out_stride + (size_t)h * lat + nt_lo * 8 + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < NT; ++n)
            if (n < my_nt) *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16(acc[n][2 * half] * inv, acc[n][2 * half + 1] * inv);
    }
}

size_t wide_smem_bytes(int lat) {
    const int pitch = lat + 8;
    return (size_t)(WR + 2 * WK) * pitch * 2 + (size_t)WR * WS_PITCH * 4 + 2 * (size_t)WR * WP_PITCH * 2 + 3 * WR * 4;
}

// out[token of seq, head, :] = sum_s acc_s e^(m_s - M) / (sum_s l_s e^(m_s - M) + e^(sink - M)), splits in ascending order.
// A lane takes a split's maximum and denominator (further ones in turn), the weights of up to MERGE_CACHED splits stay in shared
// memory (a sequence with more recomputes the rest), and a thread adds up two columns over the splits, eight loads at a time.
__global__ void __launch_bounds__(256) latent_merge_kernel(const LatParams p) {
    __shared__ float ws[MERGE_CACHED];
    __shared__ float stats[2];
    pdl_launch_dependents();
    pdl_wait();
    const int w = blockIdx.x, h = blockIdx.y, lat = p.lat;
    const int seq = p.work[w];
    const int kv_len = p.kv_len[seq];
    const int key_lo = p.window > 0 ? max(0, kv_len - p.window) : 0;
    const int n_splits = (kv_len + p.split_keys - 1) / p.split_keys - key_lo / p.split_keys;
    if ((size_t)p.split_start[w] + n_splits > (size_t)p.partial_slots) {
        if (threadIdx.x == 0) atomicOr(p.status, RS_STATUS_BAD_PLAN);
        return;
    }
    const float* base = p.partial + ((size_t)p.split_start[w] * p.n_heads + h) * (lat + 2);
    const size_t split_stride = (size_t)p.n_heads * (lat + 2);
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        float M = -INFINITY;
        for (int s = lane; s < n_splits; s += 32) M = fmaxf(M, ld_dep(base + s * split_stride + lat));
        M = warp_max(M);
        if (p.sink != nullptr) M = fmaxf(M, p.sink[h]);
        float den = p.sink != nullptr && lane == 0 ? __expf(p.sink[h] - M) : 0.f;
        for (int s = lane; s < n_splits; s += 32) {           // lane by lane, then over the lanes: a fixed order
            const float2 ml = ld_dep(reinterpret_cast<const float2*>(base + s * split_stride + lat));
            const float e = __expf(ml.x - M);
            if (s < MERGE_CACHED) ws[s] = e;
            den = fmaf(ml.y, e, den);
        }
        den = warp_sum(den);
        if (lane == 0) { stats[0] = den; stats[1] = M; }
    }
    __syncthreads();
    const float inv = 1.0f / stats[0], M = stats[1];
    __nv_bfloat16* dst = p.out + (size_t)p.q_start[seq] * p.out_stride + (size_t)h * lat;
    for (int d = 2 * threadIdx.x; d < p.v_cols; d += 2 * blockDim.x) {
        float2 num = make_float2(0.f, 0.f);
        for (int s0 = 0; s0 < n_splits; s0 += 8) {
            float2 v[8];
#pragma unroll
            for (int u = 0; u < 8; ++u)
                v[u] = s0 + u < n_splits ? ld_dep(reinterpret_cast<const float2*>(base + (s0 + u) * split_stride + d)) : make_float2(0.f, 0.f);
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                if (s0 + u >= n_splits) break;
                const float e = s0 + u < MERGE_CACHED ? ws[s0 + u] : __expf(ld_dep(base + (s0 + u) * split_stride + lat) - M);
                num.x = fmaf(v[u].x, e, num.x); num.y = fmaf(v[u].y, e, num.y);
            }
        }
        *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(num.x * inv, num.y * inv);
    }
}

size_t latent_smem_bytes(int lat, int n_buf) {
    const int pitch = lat + 8;
    return (size_t)(ROWS + n_buf * KT) * pitch * 2 + (size_t)ROWS * S_PITCH * 4 + 2 * (size_t)ROWS * P_PITCH * 2 + 3 * ROWS * 4;
}

// Two CTAs on an SM hide more than a second key buffer does: where two buffers would leave room for one CTA only
// (rows wider than about 380 values), the kernel runs with one buffer and the other CTA's work covers the loads.
constexpr size_t HALF_SM_SMEM = 113 * 1024;

// Heads whose rows a CTA of the wide kernel takes: all of them up to 64, else an equal share.
int wide_heads(int n_heads) { const int parts = (n_heads + WR - 1) / WR; return (n_heads + parts - 1) / parts; }

int heads_per_cta(int n_heads, int decode) {
    if (decode || n_heads >= ROWS) return ROWS;
    int hc = 1;
    while (hc < n_heads) hc <<= 1;
    return hc;
}
}  // namespace

RS_EXPORT int rs_attention_latent_supported(int n_heads, int lat, int page_size) {
    return n_heads > 0 && lat > 0 && lat % 16 == 0 && lat <= MAX_LAT && page_size > 0;
}

// Query tokens per work item of the portion form, narrow or wide.
RS_EXPORT int rs_attention_latent_q_per_cta(int n_heads, int wide) {
    return wide ? WR / wide_heads(n_heads) : ROWS / heads_per_cta(n_heads, 0);
}

RS_EXPORT int rs_attention_latent_bf16(const void* q, long q_stride, void* out, long out_stride, const void* cache,
                                       long page_stride, int num_pages, int page_size, const int* block_table,
                                       int table_stride, const int* q_start, const int* kv_len, const int* work, int n_work,
                                       int n_heads, int lat, int window, float scale, int decode, int split_keys,
                                       int max_splits, const int* split_start, float* partial, int partial_slots,
                                       int split_p, const float* sink, int v_cols, int wide, int* status, void* stream) {
    if (n_work <= 0) return 0;
    if (!rs_attention_latent_supported(n_heads, lat, page_size) || q_stride % 8 || out_stride % 2 || page_stride % 8 ||
        ((size_t)q & 15) || ((size_t)cache & 15) || ((size_t)out & 3))
        return (int)cudaErrorInvalidValue;
    if (v_cols <= 0 || v_cols % 8 || v_cols > lat || (wide && decode)) return (int)cudaErrorInvalidValue;
    if (decode && (split_keys % KT || split_keys <= 0 || max_splits <= 0 || partial == nullptr || partial_slots <= 0 ||
                   split_start == nullptr || ((size_t)partial & 7)))
        return (int)cudaErrorInvalidValue;
    LatParams p;
    p.q = (const __nv_bfloat16*)q; p.q_stride = q_stride; p.out = (__nv_bfloat16*)out; p.out_stride = out_stride;
    p.cache = (const __nv_bfloat16*)cache; p.page_stride = page_stride; p.num_pages = num_pages; p.page_size = page_size;
    p.block_table = block_table; p.table_stride = table_stride; p.q_start = q_start; p.kv_len = kv_len; p.work = work;
    p.n_heads = n_heads; p.lat = lat; p.hc = heads_per_cta(n_heads, decode); p.tok_per_cta = decode ? 1 : ROWS / p.hc;
    p.window = window; p.scale = scale; p.decode = decode; p.split_keys = split_keys; p.max_splits = max_splits;
    p.split_start = split_start; p.partial = partial; p.partial_slots = partial_slots; p.status = status;
    p.split_p = split_p ? 1 : 0; p.sink = sink; p.v_cols = v_cols;
    p.n_buf = latent_smem_bytes(lat, 2) <= HALF_SM_SMEM ? 2 : 1;
    const size_t smem = wide ? wide_smem_bytes(lat) : latent_smem_bytes(lat, p.n_buf);
    static std::atomic<size_t> smem_allowed[64];
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return (int)e;
    if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
    if (smem > smem_allowed[dev].load(std::memory_order_acquire)) {
        e = cudaFuncSetAttribute(latent_attention_kernel<0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_attention_kernel<8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_portion_kernel<12>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_portion_kernel<24>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        size_t seen = smem_allowed[dev].load(std::memory_order_relaxed);
        while (seen < smem && !smem_allowed[dev].compare_exchange_weak(seen, smem, std::memory_order_release)) {}
    }
    cudaStream_t s = (cudaStream_t)stream;
    if (wide) {
        p.hc = wide_heads(n_heads); p.tok_per_cta = WR / p.hc;
        const dim3 grid(n_work, (n_heads + p.hc - 1) / p.hc);
        if (((v_cols / 8 + 2) / 3 + 1) / 2 * 2 <= 12) latent_portion_kernel<12><<<grid, WTHREADS, smem, s>>>(p);
        else latent_portion_kernel<24><<<grid, WTHREADS, smem, s>>>(p);
        return rs_launch_result();
    }
    dim3 grid(n_work, (n_heads + p.hc - 1) / p.hc, decode ? max_splits : 1);
    // Wider rows read the query fragments from shared memory: kept in registers (20 or 36 steps) they cost a CTA 175 to
    // 231 registers a thread, one CTA fits an SM instead of two, and the kernel got slower (593 against 431 us for 2,048
    // tokens, 8 heads, rows of 320).
    const int rc = rs_launch_pdl(lat <= 128 ? latent_attention_kernel<8> : latent_attention_kernel<0>, grid, dim3(THREADS), smem, s, p);
    if (rc != 0 || !decode) return rc;
    return rs_launch_pdl(latent_merge_kernel, dim3(n_work, n_heads), dim3(v_cols > 256 ? 256 : 128), 0, s, p);
}
