// The experts' products of a mixture on the 5th-generation tensor cores (tcgen05 + TMEM + TMA): what moe.cu's mma.sync kernels do,
// in two shapes.  Many rows per expert: plan tiles of 128 rows, units of 256 weight rows.  Few (decoding: the products are a
// stream of weights): plan tiles of 16 rows, units of 64 weight rows, so that the units share the weights out evenly over
// the SMs, and stages of four K blocks, one 32 KB copy each (the same bytes in copies of 8 KB came at half the rate); the MMA
// still works on 128 rows, of which the others are whatever lies behind the tile.
//
// The experts' weights are packed in bands of 64 rows: [expert][band][K block][64 rows][64 columns], zeros beyond a matrix, so that a CTA
// that walks along K reads one sequential range of memory, 8 KB per K block and band.  A band of a gated unit's two matrices
// holds 32 gate rows and the 32 up rows of the same features.
//
// moe_gather:  the experts' inputs in the plan's order, row `slot` = h[token of the entry at that slot], so that the rows of an
//              expert's tile are neighbours and TMA can copy them; in column blocks, [block][slot][64 columns] (zeros beyond the
//              width), so that one copy brings several K blocks of a tile.  The activations between the products are laid out so too.  (The rows of a tile behind an expert's last one belong to
//              the next expert; their results are not stored.)
// moe_tc:      one persistent CTA per SM walks units (plan tile, column block).  Accumulators: 128 rows (lanes of tensor memory) x BR
//              columns (the unit's weight rows), two buffers, so that the epilogue of a unit runs while the next one is computed.
//              Gated units (two matrices): of every 64 columns the first 32 are gate features, the others the up values of
//              the same features, and the epilogue is the activation; else BR columns of the one matrix.
//   warp 0     TMA producer: per stage (one or four K blocks of 64) the tile's rows and BR / 64 bands of weights
//   warp 1     owns tensor memory; one thread issues the MMAs (128 x BR x 16)
//   warps 2-5  epilogue, one thread per row
// First product (MODE 1, 2, 3 as in moe_act.cuh): the activations, bfloat16; with in_weights both products' results are multiplied by
// the entry's weight first.  Second product (MODE 0): down[entry], 32-bit.
//
// Every wait is bounded; a wait that runs out sets *error_flag, and the CTA drains its copies and leaves.
#include "api.h"
#include "moe_act.cuh"
#include "tcgen05.cuh"

// ROWS: rows of a plan tile; BR: weight rows of a unit
template <int ROWS, int BR> struct mt_shape {
    static constexpr int STAGES = ROWS == 128 ? 4 : 5;
    static constexpr int KS = ROWS == 128 ? 1 : 4;     // K blocks of a stage (several only for units of one band)
    static constexpr int A_TILE = ROWS * TC_BK * 2, A_BYTES = KS * A_TILE, B_BYTES = KS * BR * TC_BK * 2;
    // the MMA reads 128 rows from the last tile's start
    static constexpr int PAD = 128 * TC_BK * 2 - A_TILE;
    static constexpr int BARS_AT = STAGES * (A_BYTES + B_BYTES) + PAD;
    static constexpr int SMEM = BARS_AT + (2 * STAGES + 4) * 8 + 16 + 1024;
    static constexpr int TMEM = 2 * BR;                // columns: two accumulators (a power of two)
};

__global__ void __launch_bounds__(256)
moe_gather_kernel(const bf16* __restrict__ h, long long ldh, const int* __restrict__ offsets, int E, const int* __restrict__ order, int top,
                  bf16* __restrict__ rows, int n_entries, int width) {
    pdl_trigger();
    pdl_wait();
    h = pdl_fresh(h);
    order = pdl_fresh(order);
    offsets = pdl_fresh(offsets);
    const int slot = blockIdx.x;
    if (slot >= offsets[E]) return;                    // (identity experts' entries have no slot)
    const bf16* src = h + (size_t)(order[slot] / top) * ldh;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    for (int i = threadIdx.x * 8; i < (width + TC_BK - 1) / TC_BK * TC_BK; i += 256 * 8)
        *reinterpret_cast<uint4*>(rows + ((size_t)(i / TC_BK) * n_entries + slot) * TC_BK + i % TC_BK) =
            i < width ? *reinterpret_cast<const uint4*>(src + i) : zero;
}

// a wait that also ends when another warp has given up
__device__ __forceinline__ bool mt_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag) {
    for (uint32_t i = 0; i < TC_WAIT_LIMIT; i++) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((i & 255) == 255 && *abort_flag) return false;
    }
    return false;
}

template <int MODE, typename TO, int ROWS, int BR>
__global__ void __launch_bounds__(TC_THREADS, 1)
moe_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b,
              const int* __restrict__ offsets, const int* __restrict__ order, const int* __restrict__ tiles, TO* __restrict__ out, long long ldo,
              int n_entries, int N, int K, int n_blocks, int bands, float limit, float alpha, const float* __restrict__ in_weights, int* __restrict__ error_flag) {
    constexpr bool GLU = MODE == 1 || MODE == 3;
    using S = mt_shape<ROWS, BR>;
    constexpr int STAGES = S::STAGES;
    constexpr int COLS = GLU ? BR / 2 : BR;            // output columns per unit
    constexpr int KS = S::KS;
    static_assert(KS == 1 || BR == 64, "several K blocks to a stage: neighbours in a band");
    static_assert(S::SMEM <= 227 * 1024 && S::TMEM >= 32 && S::TMEM <= 512 && COLS % 16 == 0, "stages or accumulators do not fit");
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    // [B stages][A stages][room behind the last A tile][barriers: full[S], empty[S], acc_full[2], acc_empty[2]]
    uint64_t* bars = (uint64_t*)(smem + S::BARS_AT);
    uint32_t* tmem_slot = (uint32_t*)(bars + 2 * STAGES + 4);
    volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
    const uint32_t b_smem = smem_u32(smem), a_smem = b_smem + STAGES * S::B_BYTES;
    const uint32_t full0 = smem_u32(bars), empty0 = smem_u32(bars + STAGES);
    const uint32_t accf0 = smem_u32(bars + 2 * STAGES), acce0 = smem_u32(bars + 2 * STAGES + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; s++) {
            mbar_init(full0 + 8 * s, 1);
            mbar_init(empty0 + 8 * s, 1);
        }
        for (int b = 0; b < 2; b++) {
            mbar_init(accf0 + 8 * b, 1);
            mbar_init(acce0 + 8 * b, 128);             // every epilogue thread
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(smem_u32(tmem_slot), S::TMEM);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_trigger();
    pdl_wait();
    offsets = pdl_fresh(offsets);
    order = pdl_fresh(order);
    tiles = pdl_fresh(tiles);
    in_weights = pdl_fresh(in_weights);
    const int units = tiles[0] * n_blocks, kb_total = (K + TC_BK - 1) / TC_BK, steps = (kb_total + KS - 1) / KS;

    if (warp == 0) {
        // ---------------------------------------------------------------- TMA producer
        if (lane == 0) {
            int g = 0;
            bool alive = true;
            for (int u = blockIdx.x; u < units && alive; u += gridDim.x) {
                const int ti = u / n_blocks, e = tiles[1 + 2 * ti], r0 = tiles[2 + 2 * ti];
                const int band0 = (u - ti * n_blocks) * (BR / 64);                   // the unit's first band of the expert's
                for (int st = 0; st < steps; st++, g++) {
                    const int s = g % STAGES;
                    if (!mt_wait(empty0 + 8 * s, ((g / STAGES) & 1) ^ 1, abort_flag)) {
                        atomicExch(error_flag, 41);
                        *abort_flag = 1;
                        alive = false;
                        break;
                    }
                    const uint32_t b = b_smem + s * S::B_BYTES, bar = full0 + 8 * s;
                    mbar_expect_tx(bar, S::A_BYTES + S::B_BYTES);
#pragma unroll
                    for (int j = 0; j < BR / 64; j++) {
                        // (a unit may reach beyond the expert's last band, and a stage beyond a band's last K block: what comes is
                        // another band's, and is not used)
                        const int band = min(band0 + j, bands - 1);
                        tma_load_2d(b + j * 64 * TC_BK * 2, &map_b, bar, 0, ((e * bands + band) * kb_total + st * KS) * 64);
                    }
                    tma_load_3d(a_smem + s * S::A_BYTES, &map_a, bar, 0, r0, st * KS);
                }
            }
            // the copies must have landed before the CTA may exit
            for (int i = max(0, g - STAGES); i < g; i++)
                if (!mbar_wait(full0 + 8 * (i % STAGES), (i / STAGES) & 1)) atomicExch(error_flag, 42);
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------------- MMA issuer
        if (lane == 0) {
            constexpr uint32_t idesc = instr_desc_bf16_mn(128, BR);
            int g = 0, item = 0;
            bool alive = true;
            for (int u = blockIdx.x; u < units && alive; u += gridDim.x, item++) {
                const int buf = item & 1;
                if (!mt_wait(acce0 + 8 * buf, ((item >> 1) & 1) ^ 1, abort_flag)) {
                    atomicExch(error_flag, 43);
                    *abort_flag = 1;
                    break;
                }
                tc_fence_after();
                const uint32_t acc = tmem_base + buf * BR;
                for (int st = 0; st < steps; st++, g++) {
                    const int s = g % STAGES;
                    if (!mt_wait(full0 + 8 * s, (g / STAGES) & 1, abort_flag)) {
                        atomicExch(error_flag, 44);
                        *abort_flag = 1;
                        alive = false;
                        break;
                    }
                    tc_fence_after();
                    const int blocks = min(KS, kb_total - st * KS);
                    for (int sub = 0; sub < blocks; sub++) {
                        const uint32_t a = a_smem + s * S::A_BYTES + sub * S::A_TILE, b = b_smem + s * S::B_BYTES + sub * (BR * TC_BK * 2);
#pragma unroll
                        for (int kk = 0; kk < TC_BK / 16; kk++)
                            umma_bf16(acc, smem_desc_sw128(a + kk * 32), smem_desc_sw128(b + kk * 32), idesc, (st | sub | kk) ? 1u : 0u);
                    }
                    umma_commit(empty0 + 8 * s);
                }
                if (alive) umma_commit(accf0 + 8 * buf);
            }
        }
    } else {
        // ---------------------------------------------------------------- epilogue: one thread per row
        const int q = warp & 3, row = q * 32 + lane;
        int item = 0;
        for (int u = blockIdx.x; u < units; u += gridDim.x, item++) {
            const int buf = item & 1;
            const int ti = u / n_blocks, n0 = (u - ti * n_blocks) * COLS;
            const int e = tiles[1 + 2 * ti], r0 = tiles[2 + 2 * ti];
            const bool here = row < ROWS && r0 + row < offsets[e + 1];     // a row of this tile and of this expert
            const int entry = here ? order[r0 + row] : 0;
            const float rw = (MODE != 0 && in_weights != nullptr && here) ? in_weights[entry] : 1.0f;
            const int slot = r0 + row, end = MODE != 0 ? (N + TC_BK - 1) / TC_BK * TC_BK : N;      // columns that are written
            // (the vote: the loads from tensor memory below are the whole warp's)
            if (!__all_sync(0xffffffffu, mt_wait(accf0 + 8 * buf, (item >> 1) & 1, abort_flag))) {
                atomicExch(error_flag, 45);
                *abort_flag = 1;
                break;
            }
            tc_fence_after();
            const uint32_t lane_addr = tmem_base + buf * BR + ((uint32_t)(q * 32) << 16);
#pragma unroll 1
            for (int c = 0; c < COLS; c += 16) {
                if (n0 + c >= end) break;                            // (the same for all)
                float v0[16], v1[16];
                const int at = GLU ? (c >> 5) * 64 + (c & 31) : c;
                tmem_ld16(lane_addr + at, v0);
                if (GLU) tmem_ld16(lane_addr + at + 32, v1);
                if (here) {
#pragma unroll
                    for (int j = 0; j < 16; j++) v0[j] = moe_first_act<MODE>(v0[j] * rw, GLU ? v1[j] * rw : 0.0f, limit, alpha);
                    if constexpr (MODE != 0) {
                        // in column blocks, as the second product reads it; zeros beyond N (a multiple of 8)
#pragma unroll
                        for (int j = 0; j < 16; j += 8) {
                            const int n = n0 + c + j;
                            if (n >= end) break;
                            uint32_t pk[4];
#pragma unroll
                            for (int k = 0; k < 4; k++) {
                                __nv_bfloat162 t = __floats2bfloat162_rn(v0[j + 2 * k], v0[j + 2 * k + 1]);
                                pk[k] = n < N ? *reinterpret_cast<uint32_t*>(&t) : 0u;
                            }
                            *reinterpret_cast<uint4*>(out + ((size_t)(n / TC_BK) * n_entries + slot) * TC_BK + n % TC_BK) =
                                make_uint4(pk[0], pk[1], pk[2], pk[3]);
                        }
                    } else {
                        TO* dst = out + (size_t)entry * ldo + n0;
#pragma unroll
                        for (int j = 0; j < 16; j += 4) {
                            if (n0 + c + j >= N) break;
                            *reinterpret_cast<float4*>(dst + c + j) = make_float4(v0[j], v0[j + 1], v0[j + 2], v0[j + 3]);
                        }
                    }
                }
            }
            tc_fence_before();
            mbar_arrive(acce0 + 8 * buf);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, S::TMEM);
    }
}

template <int MODE, typename TO, int ROWS, int BR>
static int moe_tc_launch(const void* a, int n_entries, const void* w, int n_experts, const int* offsets, const int* order,
                         const int* tiles, int max_tiles, void* out, long long ldo, int N, int K, float limit, float alpha, const float* in_weights,
                         int sms, int* error_flag, cudaStream_t s) {
    constexpr int SMEM = mt_shape<ROWS, BR>::SMEM;
    static bool done[HB_MAX_DEVICES] = {};
    if (!done[hb_device_slot()]) {
        cudaError_t e = cudaFuncSetAttribute(moe_tc_kernel<MODE, TO, ROWS, BR>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (e != cudaSuccess) return hb_fail("moe_tc: cannot reserve %d bytes of shared memory: %s", SMEM, cudaGetErrorString(e));
        done[hb_device_slot()] = true;
    }
    const int per_band = MODE == 1 || MODE == 3 ? 32 : 64, bands = (N + per_band - 1) / per_band, kbs = (K + TC_BK - 1) / TC_BK;
    const long long rows = (long long)n_experts * bands * kbs * 64;
    HB_REQUIRE(rows < (1ll << 31), "moe_tc: too many weight rows");
    CUtensorMap ma, mb;
    constexpr int KS = mt_shape<ROWS, BR>::KS;
    if (tc_make_map_blocks(&ma, a, n_entries, kbs, ROWS, KS)) return 1;
    if (tc_make_map(&mb, w, rows, TC_BK, TC_BK, 64 * KS)) return 1;
    constexpr int COLS = MODE == 1 || MODE == 3 ? BR / 2 : BR;
    // (the first product also writes the zeros up to a whole column block)
    const int columns = MODE != 0 ? (N + TC_BK - 1) / TC_BK * TC_BK : N, n_blocks = (columns + COLS - 1) / COLS;
    const long long most = (long long)max_tiles * n_blocks;
    const int grid = (int)(most < sms ? most : sms);
    cudaError_t e = hb_launch(moe_tc_kernel<MODE, TO, ROWS, BR>, dim3(grid), dim3(TC_THREADS), SMEM, s, ma, mb, offsets, order, tiles, (TO*)out, ldo, n_entries, N, K,
                              n_blocks, bands, limit, alpha, in_weights, error_flag);
    if (e != cudaSuccess) return hb_fail("moe_tc: launch failed: %s", cudaGetErrorString(e));
    return hb_check_launch("moe_tc");
}

// rows: bfloat16 [column blocks of 64][n_entries][64] of scratch, receives the experts' inputs in the plan's order
extern "C" int hb_moe_gather(const void* h, long long ldh, const int* offsets, int n_experts, const int* order, int top, void* rows, int n_entries,
                             int width, void* stream) {
    if (n_entries == 0) return 0;
    HB_REQUIRE(n_entries > 0 && width > 0 && width % 8 == 0 && top >= 1 && n_experts > 0 && ldh % 8 == 0 && (((uintptr_t)h | (uintptr_t)rows) & 15) == 0,
               "moe_gather: bfloat16 rows of a multiple of 8 elements expected");
    hb_launch(moe_gather_kernel, dim3(n_entries), dim3(256), 0, (cudaStream_t)stream, (const bf16*)h, ldh, offsets, n_experts, order, top, (bf16*)rows,
              n_entries, width);
    return hb_check_launch("moe_gather");
}

// a: bfloat16 [column blocks of K][n_entries][64] in the plan's order (tiles of tile_rows rows, 16 or 128); w: the packed
// bands of the experts' [N][K] (unit 1 and 3: of both matrices).  unit 0: out float32 [n_entries][N] at the entries' rows; 1: clamped gated
// unit, 2: exact gelu of the one matrix, 3: silu-gated unit: out bfloat16 [column blocks
// of N][n_entries][64] at the slots' rows.
extern "C" int hb_moe_tc(const void* a, int n_entries, const void* w, int n_experts, const int* offsets, const int* order,
                         const int* tiles, int max_tiles, int tile_rows, int unit, void* out, long long ldo, int N, int K, float limit, float alpha,
                         const float* in_weights, int sms, int* error_flag, void* stream) {
    if (n_entries == 0) return 0;
    HB_REQUIRE(n_entries > 0 && n_experts > 0 && max_tiles > 0 && N > 0 && K > 0 && N % 8 == 0 && K % 8 == 0 && ldo >= N && ldo % 8 == 0 && sms > 0,
               "moe_tc: bad sizes (rows of a multiple of 8 elements expected)");
    HB_REQUIRE(unit >= 0 && unit <= 3, "moe_tc: unit %d (0 to 3)", unit);
    HB_REQUIRE((((uintptr_t)a | (uintptr_t)w | (uintptr_t)out) & 15) == 0 && error_flag != nullptr, "moe_tc: operands must be 16-byte aligned");
    HB_REQUIRE(tile_rows == 16 || tile_rows == 128, "moe_tc: plan tiles of %d rows (16 or 128 are built)", tile_rows);
    cudaStream_t s = (cudaStream_t)stream;
#define HB_MT(U, TO)                                                                                                                       \
    return tile_rows == 16 ? moe_tc_launch<U, TO, 16, 64>(a, n_entries, w, n_experts, offsets, order, tiles, max_tiles, out, ldo, N, K, limit,  \
                                                          alpha, in_weights, sms, error_flag, s)                                             \
                           : moe_tc_launch<U, TO, 128, 256>(a, n_entries, w, n_experts, offsets, order, tiles, max_tiles, out, ldo, N, K,       \
                                                            limit, alpha, in_weights, sms, error_flag, s)
    if (unit == 0) HB_MT(0, float);
    if (unit == 1) HB_MT(1, bf16);
    if (unit == 2) HB_MT(2, bf16);
    HB_MT(3, bf16);
#undef HB_MT
}
