// One launch for the products of all experts of a mixture, on the warp-level tensor cores (mma.sync m16n8k16,
// bfloat16 operands, float32 accumulation): the bfloat16 engine's form of the grouped product in moe_simt.cu, with
// the same work list (moe_route: the step's (token, k) pairs sorted by expert and cut into row tiles of 16, 64 or 128).
//
// A CTA takes one row tile of one expert and a tile of rows of the expert's matrix (16 x 64, 64 x 64 or 128 x 128); it
// gathers its input rows through the sorted list (pair p reads row p / a_div of A), streams A and W in steps of k through
// several shared-memory stages with cp.async, and writes every pair's result to the pair's own row of the
// output.  Epilogues: plain store (float32 or bfloat16), or SiLU(gate) * up for a matrix whose rows
// alternate gate, up: the two lie in neighbouring accumulator columns of one thread, and the output has half the columns.
// Every output element accumulates k in ascending order, whatever else is in the batch.
#include "mma_helpers.cuh"
#include <atomic>

namespace {
// A form's tile and pipeline: BM rows x BN matrix rows a CTA, steps of BK of k, STAGES of them in shared memory, WM x WN warps.
struct Tile128 { static constexpr int BM = 128, BN = 128, BK = 32, STAGES = 4, WM = 2, WN = 4; };    // prompt portions
struct Tile64 { static constexpr int BM = 64, BN = 64, BK = 32, STAGES = 4, WM = 2, WN = 2; };       // some rows per expert
struct Tile16 { static constexpr int BM = 16, BN = 64, BK = 64, STAGES = 6, WM = 1, WN = 4; };       // single tokens

struct GroupedMmaParams {
    const void* a; int a_dt; long a_stride; int a_div;             // bfloat16, or float32 rounded to bfloat16 on the way in
    long a_expert_cols;                                            // expert e reads columns from e * a_expert_cols (0: all the same)
    const __nv_bfloat16* w; long w_expert_stride; int w_rows;      // [E][w_rows][K]
    const void* bias; int bias_dt;                                 // [E][w_rows] or null
    void* out; int out_dt; long out_stride; long out_expert_cols;  // expert e writes columns from e * out_expert_cols
    const int* order; const int* tiles; const int* n_tiles;        // tiles == null: every expert takes all dense_rows rows
    int dense_rows, tiles_per_expert;
    int K, gated;                                                  // gated: 0 plain; 1 SiLU(gate) * up of alternating rows; 2 plain, then max(., 0)^2
    OutputGate gate;                                               // GATE: the result times gate.factor(row, expert, column)
};

// 16 x 64 where an expert has a handful of rows (a decode step reads every chosen expert's matrix for them: the weights are the
// cost, fetched 128 bytes a row and step, six steps ahead), 64 x 64 for some rows, 128 x 128 for prompt portions, where the
// traffic from L2 per multiply-add halves with the tile's edge.
// GATE (plain products): the epilogue of a product behind a gate, compiled apart because it costs registers.
template <class F, bool GATE>
__global__ void __launch_bounds__(F::WM * F::WN * 32) grouped_gemm_mma_kernel(const GroupedMmaParams p) {
    constexpr int BM = F::BM, BN = F::BN, BK = F::BK, STAGES = F::STAGES, WM = F::WM, WN = F::WN, PITCH = BK + 8;
    constexpr int THREADS = WM * WN * 32, MT = BM / WM / 16, NT = BN / WN / 8, CH = BK / 8;      // CH: 16-byte columns of a step
    int e, row0, rows;
    pdl_launch_dependents();
    pdl_wait();
    if (p.tiles != nullptr) {
        if ((int)blockIdx.y >= ld_dep(p.n_tiles)) return;
        const int* tile = p.tiles + 3 * blockIdx.y;
        e = ld_dep(tile); row0 = ld_dep(tile + 1); rows = ld_dep(tile + 2);
    } else {
        e = blockIdx.y / p.tiles_per_expert;
        row0 = (blockIdx.y % p.tiles_per_expert) * BM;
        rows = min(BM, p.dense_rows - row0);
    }
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* As = reinterpret_cast<__nv_bfloat16*>(smem_raw);                  // [STAGES][BM][PITCH]
    __nv_bfloat16* Ws = As + STAGES * BM * PITCH;                                    // [STAGES][BN][PITCH]
    __shared__ int pair_of_row[BM];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int n0 = blockIdx.x * BN;
    if (tid < BM) pair_of_row[tid] = tid < rows ? (p.order != nullptr ? ld_dep(p.order + row0 + tid) : row0 + tid) : -1;
    __syncthreads();

    // a thread fetches the same 16-byte column of the same rows at every step: their addresses are found once
    constexpr int QA = BM * CH / THREADS, QW = BN * CH / THREADS;
    static_assert(THREADS % CH == 0 && QA * THREADS == BM * CH && QW * THREADS == BN * CH, "the tile's pieces divide by the threads");
    const int ch8 = (tid % CH) * 8;
    size_t a_at[QA];
    const __nv_bfloat16* w_at[QW];
    bool a_ok[QA], w_ok[QW];
#pragma unroll
    for (int q = 0; q < QA; ++q) {
        const int pr = pair_of_row[(tid + q * THREADS) / CH];
        a_ok[q] = pr >= 0;
        a_at[q] = a_ok[q] ? (size_t)(pr / p.a_div) * p.a_stride + (size_t)e * p.a_expert_cols + ch8 : 0;
    }
#pragma unroll
    for (int q = 0; q < QW; ++q) {
        const int gn = n0 + (tid + q * THREADS) / CH;
        w_ok[q] = gn < p.w_rows;
        w_at[q] = p.w + (size_t)e * p.w_expert_stride + (w_ok[q] ? (size_t)gn * p.K + ch8 : 0);
    }
    auto load = [&](int stage, int k0) {
        const bool k_ok = k0 + ch8 < p.K;
#pragma unroll
        for (int q = 0; q < QA; ++q) {
            __nv_bfloat16* dst = As + (stage * BM + (tid + q * THREADS) / CH) * PITCH + ch8;
            if (a_ok[q] && k_ok) {
                if (p.a_dt == RS_BF16) {
                    cp_async16(smem_addr(dst), reinterpret_cast<const __nv_bfloat16*>(p.a) + a_at[q] + k0);
                } else {
                    const float* src = reinterpret_cast<const float*>(p.a) + a_at[q] + k0;
                    const float4 lo = ld_dep(reinterpret_cast<const float4*>(src)), hi = ld_dep(reinterpret_cast<const float4*>(src + 4));
                    uint4 u;
                    u.x = pack_bf16(lo.x, lo.y); u.y = pack_bf16(lo.z, lo.w); u.z = pack_bf16(hi.x, hi.y); u.w = pack_bf16(hi.z, hi.w);
                    *reinterpret_cast<uint4*>(dst) = u;
                }
            } else {
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
            }
        }
#pragma unroll
        for (int q = 0; q < QW; ++q) {
            __nv_bfloat16* dst = Ws + (stage * BN + (tid + q * THREADS) / CH) * PITCH + ch8;
            if (w_ok[q] && k_ok) cp_async16(smem_addr(dst), w_at[q] + k0);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
    };

    float acc[MT][NT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NT; ++j) { acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f; }
    const int m_base = (warp / WN) * (BM / WM), n_base = (warp % WN) * (BN / WN);
    const int a_row = (lane & 7) + 8 * ((lane >> 3) & 1), a_col = 8 * (lane >> 4);
    const int b_row = (lane & 7) + 8 * (lane >> 4), b_col = 8 * ((lane >> 3) & 1);
    const int n_steps = (p.K + BK - 1) / BK;
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) {
        if (s < n_steps) load(s, s * BK);
        cp_async_commit();
    }
    for (int s = 0; s < n_steps; ++s) {
        cp_async_wait<STAGES - 2>();
        __syncthreads();                           // step s is here; nobody reads the stage of step s - 1 any more
        if (s + STAGES - 1 < n_steps) load((s + STAGES - 1) % STAGES, (s + STAGES - 1) * BK);
        cp_async_commit();
        const __nv_bfloat16* At = As + (s % STAGES) * BM * PITCH;
        const __nv_bfloat16* Wt = Ws + (s % STAGES) * BN * PITCH;
#pragma unroll
        for (int kk = 0; kk < BK; kk += 16) {
            uint32_t a[MT][4], b[NT][2];
#pragma unroll
            for (int i = 0; i < MT; ++i)
                ldmatrix_x4(smem_addr(At + (m_base + i * 16 + a_row) * PITCH + kk + a_col), a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
            for (int j = 0; j < NT / 2; ++j)
                ldmatrix_x4(smem_addr(Wt + (n_base + j * 16 + b_row) * PITCH + kk + b_col), b[2 * j][0], b[2 * j][1], b[2 * j + 1][0],
                            b[2 * j + 1][1]);
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int j = 0; j < NT; ++j) mma16816(acc[i][j], a[i], b[j][0], b[j][1]);
        }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int pr = pair_of_row[m_base + i * 16 + (lane >> 2) + 8 * half];
            if (pr < 0) continue;
            const bool row_gate = GATE && (p.gate.g == nullptr || p.gate.per_block);
            const float row_factor = row_gate ? p.gate.factor(pr, e, 0) : 1.0f;
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int gn = n0 + n_base + j * 8 + (lane & 3) * 2;
                float c0 = acc[i][j][2 * half], c1 = acc[i][j][2 * half + 1];
                if (p.bias != nullptr) {
                    if (gn < p.w_rows) c0 += load_any(p.bias, p.bias_dt, (size_t)e * p.w_rows + gn);
                    if (gn + 1 < p.w_rows) c1 += load_any(p.bias, p.bias_dt, (size_t)e * p.w_rows + gn + 1);
                }
                if (p.gated == 2) {
                    c0 = fmaxf(c0, 0.f); c0 *= c0;
                    c1 = fmaxf(c1, 0.f); c1 *= c1;
                }
                if (GATE) {
                    c0 *= row_gate ? row_factor : gn < p.w_rows ? p.gate.factor(pr, e, e * p.w_rows + gn) : 0.f;
                    c1 *= row_gate ? row_factor : gn + 1 < p.w_rows ? p.gate.factor(pr, e, e * p.w_rows + gn + 1) : 0.f;
                }
                if (p.gated == 1) {
                    if (gn + 1 < p.w_rows) {
                        const float v = silu_mul_fast(c0, c1);
                        const size_t o = (size_t)pr * p.out_stride + (size_t)e * p.out_expert_cols + (gn >> 1);
                        if (p.out_dt == RS_F32) reinterpret_cast<float*>(p.out)[o] = v;
                        else reinterpret_cast<__nv_bfloat16*>(p.out)[o] = __float2bfloat16_rn(v);
                    }
                } else {
                    const size_t o = (size_t)pr * p.out_stride + (size_t)e * p.out_expert_cols + gn;
                    if (p.out_dt == RS_F32) {
                        float* dst = reinterpret_cast<float*>(p.out) + o;
                        if (gn < p.w_rows) dst[0] = c0;
                        if (gn + 1 < p.w_rows) dst[1] = c1;
                    } else {
                        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + o;
                        if (gn < p.w_rows) dst[0] = __float2bfloat16_rn(c0);
                        if (gn + 1 < p.w_rows) dst[1] = __float2bfloat16_rn(c1);
                    }
                }
            }
        }
}

// Launches a form for ``row_tiles`` tiles of rows (times blocks).
template <class F, bool GATE>
int launch_grouped(const GroupedMmaParams& p, int row_tiles, cudaStream_t s) {
    constexpr size_t smem = (size_t)F::STAGES * (F::BM + F::BN) * (F::BK + 8) * sizeof(__nv_bfloat16);
    auto kern = grouped_gemm_mma_kernel<F, GATE>;
    if (smem > 48 * 1024) {                        // the opt-in is a property of (kernel, device): asked for once on each
        static std::atomic<bool> allowed[64];
        int dev = 0;
        cudaError_t e = cudaGetDevice(&dev);
        if (e != cudaSuccess) return (int)e;
        if (dev < 0 || dev >= 64) return (int)cudaErrorInvalidDevice;
        if (!allowed[dev].load(std::memory_order_acquire)) {
            e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
            allowed[dev].store(true, std::memory_order_release);
        }
    }
    return rs_launch_pdl(kern, dim3((p.w_rows + F::BN - 1) / F::BN, row_tiles), dim3(F::WM * F::WN * 32), smem, s, p);
}
}  // namespace

// Rows of one expert per CTA of form 0 (single tokens), 1 (some rows per expert) and 2 (prompt portions).
RS_EXPORT int rs_grouped_gemm_mma_rows_per_tile(int form) { return form == 2 ? Tile128::BM : form == 1 ? Tile64::BM : Tile16::BM; }

// a: bfloat16 [*, K] rows 16-byte aligned; w: bfloat16 [E][w_rows][K]; out: [pairs, w_rows] (or w_rows / 2 when gated,
// the rows of w alternating gate, up).  K a multiple of 8.
RS_EXPORT int rs_grouped_gemm_mma(const void* a, long a_stride, int a_div, const void* w, long w_expert_stride, int w_rows,
                                  void* out, int out_dt, long out_stride, const int* order, const int* tiles,
                                  const int* n_tiles, int max_tiles, int K, int gated, int form, void* stream) {
    if (max_tiles <= 0 || w_rows <= 0) return 0;
    if (K <= 0 || K % 8 || a_stride % 8 || w_expert_stride % 8 || ((size_t)a & 15) || ((size_t)w & 15) || (gated == 1 && w_rows % 2) || gated < 0 || gated > 2 || form < 0 || form > 2)
        return (int)cudaErrorInvalidValue;
    GroupedMmaParams p{a, RS_BF16, a_stride, a_div, 0, (const __nv_bfloat16*)w, w_expert_stride, w_rows, nullptr, 0, out, out_dt,
                       out_stride, 0, order, tiles, n_tiles, 0, 1, K, gated, OutputGate{nullptr, 0, 0, 1.0f}};
    const cudaStream_t s = (cudaStream_t)stream;
    if (form == 2) return launch_grouped<Tile128, false>(p, max_tiles, s);
    return form == 1 ? launch_grouped<Tile64, false>(p, max_tiles, s) : launch_grouped<Tile16, false>(p, max_tiles, s);
}

// The block-diagonal product of sequence_parts.cu (rs_block_linear) for more than a few rows, through the same kernel:
// block b is an "expert" that takes every row, reads columns from b * in_bs and writes columns from b * out_bs.
//   out[t, b * out_bs + o] = (bias[b, o] + sum_i W[b, o, i] * x[t, b * in_bs + i]) * out_scale * sigmoid(gate)
// (gate as in rs_block_linear; null: none).
// x: bfloat16, or float32 (rounded to bfloat16 as it enters the product); W: bfloat16 [B, O, I], I a multiple of 8.
RS_EXPORT int rs_block_linear_mma(const void* x, int x_dt, long x_stride, long in_bs, const void* w, const void* bias,
                                  int bias_dt, void* out, int out_dt, long out_stride, long out_bs, int T, int B, int O,
                                  int I, const float* gate, long gate_stride, int gate_per_block, float out_scale, void* stream) {
    if (T <= 0 || B <= 0 || O <= 0) return 0;
    const int align = x_dt == RS_F32 ? 4 : 8;                  // elements per 16 bytes
    if (I <= 0 || I % 8 || x_stride % align || in_bs % align || ((size_t)x & 15) || ((size_t)w & 15))
        return (int)cudaErrorInvalidValue;
    const int bm = T > 256 ? 128 : 64;
    const int tiles_per = (T + bm - 1) / bm;
    GroupedMmaParams p{x, x_dt, x_stride, 1, in_bs, (const __nv_bfloat16*)w, (long)O * I, O, bias, bias_dt, out, out_dt, out_stride,
                       out_bs, nullptr, nullptr, nullptr, T, tiles_per, I, 0, OutputGate{gate, gate_stride, gate_per_block, out_scale}};
    const cudaStream_t s = (cudaStream_t)stream;
    if (gate != nullptr || out_scale != 1.0f)
        return bm == 128 ? launch_grouped<Tile128, true>(p, tiles_per * B, s) : launch_grouped<Tile64, true>(p, tiles_per * B, s);
    return bm == 128 ? launch_grouped<Tile128, false>(p, tiles_per * B, s) : launch_grouped<Tile64, false>(p, tiles_per * B, s);
}
