// The experts' products of a mixture on the 5th-generation tensor cores (tcgen05 + TMEM + TMA), for steps that bring many
// tokens: what moe.cu's mma.sync kernels do, over plan tiles of 128 rows.
//
// moe_gather:  rows[slot] = h[token of the entry at that slot]: the experts' inputs in the plan's order, so that the rows of an
//              expert's tile are neighbours and TMA can copy them.  (The rows of a tile behind an expert's last one belong to
//              the next expert; their results are not stored.)
// moe_tc:      one persistent CTA per SM walks units (plan tile, column block).  Accumulators: 128 rows (lanes of tensor memory) x 256
//              columns, two buffers, so that the epilogue of a unit runs while the next one is computed.  Gated units (two
//              matrices): columns 0..127 are gate features, 128..255 the up values of the same features, and the epilogue is
//              the activation; else 256 columns of the one matrix.
//   warp 0     TMA producer: per K block of 64 the tile's rows (16 KB) and twice 128 weight rows (32 KB), four stages
//   warp 1     owns tensor memory; one thread issues the MMAs (128 x 256 x 16)
//   warps 2-5  epilogue, one thread per row
// First product (MODE 1, 2, 3 as in moe_act.cuh): act[slot], bfloat16; with in_weights both products' results are multiplied by
// the entry's weight first.  Second product (MODE 0): down[entry], 32-bit.
//
// Every wait is bounded; a wait that runs out sets *error_flag, and the CTA drains its copies and leaves.
#include "api.h"
#include "moe_act.cuh"
#include "tcgen05.cuh"

#define MT_ROWS 128
#define MT_STAGES 4
#define MT_A_BYTES (MT_ROWS * TC_BK * 2)               // 16 KB
#define MT_B_BYTES (2 * 128 * TC_BK * 2)               // 32 KB
#define MT_STAGE_BYTES (MT_A_BYTES + MT_B_BYTES)
#define MT_SMEM (MT_STAGES * MT_STAGE_BYTES + (2 * MT_STAGES + 4) * 8 + 16 + 1024)

__global__ void __launch_bounds__(256)
moe_gather_kernel(const bf16* __restrict__ h, long long ldh, const int* __restrict__ offsets, int E, const int* __restrict__ order, int top,
                  bf16* __restrict__ rows, int width) {
    pdl_trigger();
    pdl_wait();
    h = pdl_fresh(h);
    order = pdl_fresh(order);
    offsets = pdl_fresh(offsets);
    const int slot = blockIdx.x;
    if (slot >= offsets[E]) return;                    // (identity experts' entries have no slot)
    const bf16* src = h + (size_t)(order[slot] / top) * ldh;
    bf16* dst = rows + (size_t)slot * width;
    for (int i = threadIdx.x * 8; i < width; i += 256 * 8) *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<const uint4*>(src + i);
}

// a wait that also ends when another warp has given up
__device__ __forceinline__ bool mt_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag) {
    for (uint32_t i = 0; i < TC_WAIT_LIMIT; i++) {
        if (mbar_try_wait(bar, parity)) return true;
        if ((i & 255) == 255 && *abort_flag) return false;
    }
    return false;
}

template <int MODE, typename TO>
__global__ void __launch_bounds__(TC_THREADS, 1)
moe_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b0, const __grid_constant__ CUtensorMap map_b1,
              const int* __restrict__ offsets, const int* __restrict__ order, const int* __restrict__ tiles, TO* __restrict__ out, long long ldo,
              int N, int K, int n_blocks, float limit, float alpha, const float* __restrict__ in_weights, int* __restrict__ error_flag) {
    constexpr bool GLU = MODE == 1 || MODE == 3;
    constexpr int COLS = GLU ? 128 : 256;              // output columns per unit
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint64_t* bars = (uint64_t*)(smem + MT_STAGES * MT_STAGE_BYTES);       // full[S], empty[S], acc_full[2], acc_empty[2]
    uint32_t* tmem_slot = (uint32_t*)(bars + 2 * MT_STAGES + 4);
    volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
    const uint32_t smem_base = smem_u32(smem);
    const uint32_t full0 = smem_u32(bars), empty0 = smem_u32(bars + MT_STAGES);
    const uint32_t accf0 = smem_u32(bars + 2 * MT_STAGES), acce0 = smem_u32(bars + 2 * MT_STAGES + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int s = 0; s < MT_STAGES; s++) {
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
    if (warp == 1) tmem_alloc(smem_u32(tmem_slot), 512);
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
    const int units = tiles[0] * n_blocks, kb_total = (K + TC_BK - 1) / TC_BK;

    if (warp == 0) {
        // ---------------------------------------------------------------- TMA producer
        if (lane == 0) {
            int g = 0;
            bool alive = true;
            for (int u = blockIdx.x; u < units && alive; u += gridDim.x) {
                const int ti = u / n_blocks, n0 = (u - ti * n_blocks) * COLS;
                const int e = tiles[1 + 2 * ti], r0 = tiles[2 + 2 * ti];
                const int w_row = e * N + n0;
                for (int kb = 0; kb < kb_total; kb++, g++) {
                    const int s = g % MT_STAGES;
                    if (!mt_wait(empty0 + 8 * s, ((g / MT_STAGES) & 1) ^ 1, abort_flag)) {
                        atomicExch(error_flag, 41);
                        *abort_flag = 1;
                        alive = false;
                        break;
                    }
                    const uint32_t stage = smem_base + s * MT_STAGE_BYTES, bar = full0 + 8 * s;
                    mbar_expect_tx(bar, MT_STAGE_BYTES);
                    tma_load_2d(stage, &map_a, bar, kb * TC_BK, r0);
                    tma_load_2d(stage + MT_A_BYTES, &map_b0, bar, kb * TC_BK, w_row);
                    if (GLU) tma_load_2d(stage + MT_A_BYTES + MT_B_BYTES / 2, &map_b1, bar, kb * TC_BK, w_row);
                    else tma_load_2d(stage + MT_A_BYTES + MT_B_BYTES / 2, &map_b0, bar, kb * TC_BK, w_row + 128);
                }
            }
            // the copies must have landed before the CTA may exit
            for (int i = max(0, g - MT_STAGES); i < g; i++)
                if (!mbar_wait(full0 + 8 * (i % MT_STAGES), (i / MT_STAGES) & 1)) atomicExch(error_flag, 42);
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------------- MMA issuer
        if (lane == 0) {
            constexpr uint32_t idesc = instr_desc_bf16_mn(128, 256);
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
                const uint32_t acc = tmem_base + buf * 256;
                for (int kb = 0; kb < kb_total; kb++, g++) {
                    const int s = g % MT_STAGES;
                    if (!mt_wait(full0 + 8 * s, (g / MT_STAGES) & 1, abort_flag)) {
                        atomicExch(error_flag, 44);
                        *abort_flag = 1;
                        alive = false;
                        break;
                    }
                    tc_fence_after();
                    const uint32_t a = smem_base + s * MT_STAGE_BYTES, b = a + MT_A_BYTES;
#pragma unroll
                    for (int kk = 0; kk < TC_BK / 16; kk++)
                        umma_bf16(acc, smem_desc_sw128(a + kk * 32), smem_desc_sw128(b + kk * 32), idesc, (kb | kk) ? 1u : 0u);
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
            const bool here = r0 + row < offsets[e + 1];
            const int entry = here ? order[r0 + row] : 0;
            const float rw = (MODE != 0 && in_weights != nullptr && here) ? in_weights[entry] : 1.0f;
            TO* dst = out + (size_t)(MODE != 0 ? r0 + row : entry) * ldo + n0;
            // (the vote: the loads from tensor memory below are the whole warp's)
            if (!__all_sync(0xffffffffu, mt_wait(accf0 + 8 * buf, (item >> 1) & 1, abort_flag))) {
                atomicExch(error_flag, 45);
                *abort_flag = 1;
                break;
            }
            tc_fence_after();
            const uint32_t lane_addr = tmem_base + buf * 256 + ((uint32_t)(q * 32) << 16);
#pragma unroll 1
            for (int c = 0; c < COLS; c += 16) {
                if (n0 + c >= N) break;                              // (the same for all)
                float v0[16], v1[16];
                tmem_ld16(lane_addr + c, v0);
                if (GLU) tmem_ld16(lane_addr + 128 + c, v1);
                if (here) {
#pragma unroll
                    for (int j = 0; j < 16; j++) v0[j] = moe_first_act<MODE>(v0[j] * rw, GLU ? v1[j] * rw : 0.0f, limit, alpha);
                    if constexpr (sizeof(TO) == 2) {
#pragma unroll
                        for (int j = 0; j < 16; j += 8) {
                            if (n0 + c + j >= N) break;              // (N is a multiple of 8)
                            uint32_t pk[4];
#pragma unroll
                            for (int k = 0; k < 4; k++) {
                                __nv_bfloat162 t = __floats2bfloat162_rn(v0[j + 2 * k], v0[j + 2 * k + 1]);
                                pk[k] = *reinterpret_cast<uint32_t*>(&t);
                            }
                            *reinterpret_cast<uint4*>(dst + c + j) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                        }
                    } else {
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
        tmem_dealloc(tmem_base, 512);
    }
}

template <int MODE, typename TO>
static int moe_tc_launch(const CUtensorMap& ma, const CUtensorMap& m0, const CUtensorMap& m1, const int* offsets, const int* order, const int* tiles,
                         int max_tiles, void* out, long long ldo, int N, int K, float limit, float alpha, const float* in_weights, int sms,
                         int* error_flag, cudaStream_t s) {
    static bool done[HB_MAX_DEVICES] = {};
    if (!done[hb_device_slot()]) {
        cudaError_t e = cudaFuncSetAttribute(moe_tc_kernel<MODE, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, MT_SMEM);
        if (e != cudaSuccess) return hb_fail("moe_tc: cannot reserve %d bytes of shared memory: %s", MT_SMEM, cudaGetErrorString(e));
        done[hb_device_slot()] = true;
    }
    constexpr int COLS = MODE == 1 || MODE == 3 ? 128 : 256;
    const int n_blocks = (N + COLS - 1) / COLS;
    const long long most = (long long)max_tiles * n_blocks;
    const int grid = (int)(most < sms ? most : sms);
    cudaError_t e = hb_launch(moe_tc_kernel<MODE, TO>, dim3(grid), dim3(TC_THREADS), MT_SMEM, s, ma, m0, m1, offsets, order, tiles, (TO*)out, ldo, N, K,
                              n_blocks, limit, alpha, in_weights, error_flag);
    if (e != cudaSuccess) return hb_fail("moe_tc: launch failed: %s", cudaGetErrorString(e));
    return hb_check_launch("moe_tc");
}

// rows: bfloat16 [n_entries][width] of scratch, receives the experts' inputs in the plan's order
extern "C" int hb_moe_gather(const void* h, long long ldh, const int* offsets, int n_experts, const int* order, int top, void* rows, int n_entries,
                             int width, void* stream) {
    if (n_entries == 0) return 0;
    HB_REQUIRE(n_entries > 0 && width > 0 && width % 8 == 0 && top >= 1 && n_experts > 0 && ldh % 8 == 0 && (((uintptr_t)h | (uintptr_t)rows) & 15) == 0,
               "moe_gather: bfloat16 rows of a multiple of 8 elements expected");
    hb_launch(moe_gather_kernel, dim3(n_entries), dim3(256), 0, (cudaStream_t)stream, (const bf16*)h, ldh, offsets, n_experts, order, top, (bf16*)rows, width);
    return hb_check_launch("moe_gather");
}

// a: bfloat16 [n_entries][K] in the plan's order (tiles of 128 rows); w0, w1: bfloat16 stacks [n_experts][N][K] (w1 null: one matrix).  unit 0: out
// float32 [n_entries][N] at the entries' rows; 1: clamped gated unit, 2: exact gelu of w0, 3: silu-gated unit: out bfloat16 at the slots' rows.
extern "C" int hb_moe_tc(const void* a, int n_entries, const void* w0, const void* w1, int n_experts, const int* offsets, const int* order,
                         const int* tiles, int max_tiles, int unit, void* out, long long ldo, int N, int K, float limit, float alpha,
                         const float* in_weights, int sms, int* error_flag, void* stream) {
    if (n_entries == 0) return 0;
    HB_REQUIRE(n_entries > 0 && n_experts > 0 && max_tiles > 0 && N > 0 && K > 0 && N % 8 == 0 && K % 8 == 0 && ldo >= N && ldo % 8 == 0 && sms > 0,
               "moe_tc: bad sizes (rows of a multiple of 8 elements expected)");
    HB_REQUIRE((long long)n_experts * N < (1ll << 31), "moe_tc: too many weight rows");
    HB_REQUIRE(unit >= 0 && unit <= 3 && (w1 != nullptr) == (unit == 1 || unit == 3), "moe_tc: unit %d (1 and 3: two matrices, 0 and 2: one)", unit);
    HB_REQUIRE((((uintptr_t)a | (uintptr_t)w0 | (uintptr_t)w1 | (uintptr_t)out) & 15) == 0 && error_flag != nullptr, "moe_tc: operands must be 16-byte aligned");
    CUtensorMap ma, m0, m1;
    if (tc_make_map(&ma, a, n_entries, K, K, MT_ROWS)) return 1;
    if (tc_make_map(&m0, w0, (long long)n_experts * N, K, K, 128)) return 1;
    if (tc_make_map(&m1, w1 != nullptr ? w1 : w0, (long long)n_experts * N, K, K, 128)) return 1;
    cudaStream_t s = (cudaStream_t)stream;
#define HB_MT(U, TO) return moe_tc_launch<U, TO>(ma, m0, m1, offsets, order, tiles, max_tiles, out, ldo, N, K, limit, alpha, in_weights, sms, error_flag, s)
    if (unit == 0) HB_MT(0, float);
    if (unit == 1) HB_MT(1, bf16);
    if (unit == 2) HB_MT(2, bf16);
    HB_MT(3, bf16);
#undef HB_MT
}
