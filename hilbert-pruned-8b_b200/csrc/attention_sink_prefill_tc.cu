// Softmax attention for steps that bring many tokens, on the 5th-generation tensor cores (tcgen05 + TMEM + TMA): what
// attention_sink_prefill.cu does with mma.sync, for heads whose softmax weights are not mixed.  Causal, grouped-query, with a
// sliding window or chunks of positions, a sink, key and value heads of different sizes, a gate on the results (per head or
// per element) and columns of ones behind them, over the paged bfloat16 cache, for batches of sequences with unequal numbers
// of new tokens.
//
// One CTA = 128 consecutive new tokens of one sequence x one query head, in the roles of attention_prefill_tc.cu:
//   warp 0     TMA producer (the query tile, then tiles of 128 keys and of 128 values, freed separately)
//   warp 1     owns tensor memory; one thread issues the MMAs: S_j = Q K_j^T, then O += P_j V_j with P_j in tensor memory
//   warps 2-9  softmax, two threads per query row (64 key columns each), and the output
// The softmax weights stay exact to 16 mantissa bits: P_j is written over S_j as TWO bfloat16 terms, hi = bf16(p) in columns
// 0..63 and lo = bf16(p - hi) in columns 64..127 of the tile's 128, and both meet the same values (two MMAs per 16 keys).
// Scores, running maximum, sum and the output accumulator are float32; the normalised result is multiplied by the gate in
// float32 and rounded once.
//
// Head sizes are any multiple of 8 up to HDP (keys: 64, 128, 192) and VDP (values: 64, 128): the tensor maps of the cache end
// at the head's size, so the copies fill the rest of a 64-column box with zeros.  (The query box may reach into the next head's
// columns; they meet the keys' zeros.)
//
// Every wait is bounded; a wait that runs out sets *error_flag and the CTA drains and leaves.
#include "api.h"
#include "attention_tc.cuh"

// stages of key tiles and of value tiles: what fits beside the query tile
template <int HDP> struct st_stages { static constexpr int N = HDP <= 128 ? 3 : 2; };

template <int HDP, int VDP>
__global__ void __launch_bounds__(FA_THREADS, 1)
attn_sink_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                            const __grid_constant__ CUtensorMap map_v, const int* __restrict__ page_table, int pt_width,
                            const int* __restrict__ seq_start, const int* __restrict__ seq_pos0, bf16* __restrict__ out, long long out_stride,
                            int ones, const float* __restrict__ gate, long long ldg, int gate_per, int n_seqs, int nh, int nkv, int hd, int vd,
                            float scale_log2e, int window, int chunk, const float* __restrict__ sink, int n_pages, int* __restrict__ error_flag) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    // [Q tile][K stages][V stages][barriers]; a tile is 128 rows x HDP (or VDP), in sub-tiles of 64 columns
    constexpr int STAGES = st_stages<HDP>::N;
    constexpr int K_TILE = HDP / 64 * FA_HALF_BYTES, V_TILE = VDP / 64 * FA_HALF_BYTES;
    uint64_t* bars = (uint64_t*)(smem + K_TILE + STAGES * (K_TILE + V_TILE));
    uint32_t* tmem_slot = (uint32_t*)(bars + 18);
    volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
    float* xrow = (float*)(tmem_slot + 4);                    // [2 halves][128 rows]: row maxima, at the end row sums
    const uint32_t smem_base = smem_u32(smem);
    const uint32_t k_smem = smem_base + K_TILE, v_smem = k_smem + STAGES * K_TILE;
    const uint32_t q_full = smem_u32(bars), k_full0 = smem_u32(bars + 1), k_empty0 = smem_u32(bars + 4);
    const uint32_t v_full0 = smem_u32(bars + 7), v_empty0 = smem_u32(bars + 10);
    const uint32_t s_full0 = smem_u32(bars + 13), p_full0 = smem_u32(bars + 15), pv_done = smem_u32(bars + 17);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x, g = head / (nh / nkv);

    // which sequence and which block of its new tokens: blocks from the back, heads fastest, so that the query blocks that see
    // the most keys start first
    int b = 0, blk = gridDim.y - 1 - blockIdx.y;
    for (; b < n_seqs; b++) {
        const int nb = (seq_start[b + 1] - seq_start[b] + FA_ROWS - 1) / FA_ROWS;
        if (blk < nb) break;
        blk -= nb;
    }
    const bool has_work = b < n_seqs;
    const int t_begin = has_work ? seq_start[b] : 0, n_new = has_work ? seq_start[b + 1] - t_begin : 0;
    const int pos0 = has_work ? seq_pos0[b] : 0;
    const int row_base = blk * FA_ROWS;
    const int rows_here = min(FA_ROWS, n_new - row_base);
    const int first_pos = pos0 + row_base, last_pos = first_pos + rows_here - 1;
    const int lo_cta = hb_oldest_visible(first_pos, window, chunk);
    const int jt0 = lo_cta / FA_KEYS, jt1 = has_work ? last_pos / FA_KEYS + 1 : 0;
    const int n_it = jt1 - jt0;

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int s = 0; s < STAGES; s++) {
            mbar_init(k_full0 + 8 * s, 1);
            mbar_init(k_empty0 + 8 * s, 1);
            mbar_init(v_full0 + 8 * s, 1);
            mbar_init(v_empty0 + 8 * s, 1);
        }
        for (int s = 0; s < 2; s++) {
            mbar_init(s_full0 + 8 * s, 1);
            mbar_init(p_full0 + 8 * s, 256);
        }
        mbar_init(pv_done, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(smem_u32(tmem_slot), 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t tm_o = tmem_base + 256;               // S buffers at columns 0 and 128, O at 256
    pdl_trigger();
    pdl_wait();                                          // queries, keys and values come from the kernels in front
    gate = pdl_fresh(gate);

    if (warp == 0) {
        // ---------------------------------------------------------------- TMA producer
        if (lane == 0 && n_it > 0) {
            const int* pt = page_table + (size_t)b * pt_width;
            mbar_expect_tx(q_full, K_TILE);
            for (int sub = 0; sub < HDP / 64; sub++)
                tma_load_2d(smem_base + sub * FA_HALF_BYTES, &map_q, q_full, head * hd + sub * 64, t_begin + row_base);
            auto load_tile = [&](uint32_t dst, const CUtensorMap* map, uint32_t bar, int it, int subs) {
                mbar_expect_tx(bar, subs * FA_HALF_BYTES);
                for (int pg = 0; pg < 2; pg++) {
                    const int pi = (jt0 + it) * 2 + pg;
                    int page = pi < pt_width ? pt[pi] : -1;
                    if (page < 0 || page >= n_pages) {
                        // a tile's second page may lie behind the sequence's end, and its first one in front of the window
                        // (their keys are masked); a page between the oldest key the first row sees and the last row's own
                        // key must exist: the host's bookkeeping is at fault
                        if (page >= n_pages || (pi >= lo_cta / HB_PAGE_TOKENS && pi <= last_pos / HB_PAGE_TOKENS))
                            hb_note(error_flag, HB_STATUS_PAGE, 1 + b);
                        page = 0;                                   // never read outside the cache
                    }
                    const int row = (page * nkv + g) * HB_PAGE_TOKENS;
                    for (int sub = 0; sub < subs; sub++)
                        tma_load_2d(dst + sub * FA_HALF_BYTES + pg * (FA_HALF_BYTES / 2), map, bar, sub * 64, row);
                }
            };
            int k_issued = 0, v_issued = 0;
            bool alive = true;
            for (int step = 0; step < n_it + 1 && alive; step++) {
                const int ik = step, iv = step - 1;                 // the keys of tile `step`, then the values of the tile before
                if (ik < n_it) {
                    const int s = ik % STAGES;
                    if (!mbar_wait(k_empty0 + 8 * s, ((ik / STAGES) & 1) ^ 1)) {
                        atomicExch(error_flag, 21);
                        *abort_flag = 1;
                        alive = false;
                        break;
                    }
                    load_tile(k_smem + s * K_TILE, &map_k, k_full0 + 8 * s, ik, HDP / 64);
                    k_issued = ik + 1;
                }
                if (iv >= 0) {
                    const int s = iv % STAGES;
                    if (!mbar_wait(v_empty0 + 8 * s, ((iv / STAGES) & 1) ^ 1)) {
                        atomicExch(error_flag, 22);
                        *abort_flag = 1;
                        alive = false;
                        break;
                    }
                    load_tile(v_smem + s * V_TILE, &map_v, v_full0 + 8 * s, iv, VDP / 64);
                    v_issued = iv + 1;
                }
            }
            for (int it = max(0, k_issued - STAGES); it < k_issued; it++)
                if (!mbar_wait(k_full0 + 8 * (it % STAGES), (it / STAGES) & 1)) atomicExch(error_flag, 23);
            for (int it = max(0, v_issued - STAGES); it < v_issued; it++)
                if (!mbar_wait(v_full0 + 8 * (it % STAGES), (it / STAGES) & 1)) atomicExch(error_flag, 23);
            if (!mbar_wait(q_full, 0)) atomicExch(error_flag, 23);
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------------- MMA issuer
        if (lane == 0 && n_it > 0) {
            constexpr uint32_t idesc_qk = instr_desc_bf16_mn(128, FA_KEYS);
            constexpr uint32_t idesc_pv = instr_desc_bf16_mn(128, VDP) | (1u << 16);          // B is MN-major
            const int ksteps = (hd + 15) / 16;
            bool alive = mbar_wait(q_full, 0);
            if (!alive) { atomicExch(error_flag, 24); *abort_flag = 1; }
            auto issue_qk = [&](int it) {
                const int s = it % STAGES, sb = it & 1;
                if (!mbar_wait(k_full0 + 8 * s, (it / STAGES) & 1)) {
                    atomicExch(error_flag, 25);
                    *abort_flag = 1;
                    alive = false;
                    return;
                }
                tc_fence_after();
                const uint32_t kst = k_smem + s * K_TILE;
#pragma unroll 4
                for (int kk = 0; kk < ksteps; kk++) {
                    const uint32_t off = (kk >> 2) * FA_HALF_BYTES + (kk & 3) * 32;
                    umma_bf16(tmem_base + sb * 128, smem_desc_sw128(smem_base + off), smem_desc_sw128(kst + off), idesc_qk, kk ? 1u : 0u);
                }
                umma_commit(k_empty0 + 8 * s);                // the key tile is used up
                umma_commit(s_full0 + 8 * sb);
            };
            if (alive) issue_qk(0);
            for (int it = 0; it < n_it && alive; it++) {
                const int s = it & 1;
                if (it + 1 < n_it) issue_qk(it + 1);          // runs while the softmax warps work on tile `it`
                if (!alive) break;
                if (!mbar_wait(p_full0 + 8 * s, (it >> 1) & 1)) {
                    atomicExch(error_flag, 26);
                    *abort_flag = 1;
                    break;
                }
                const int sv = it % STAGES;
                if (!mbar_wait(v_full0 + 8 * sv, (it / STAGES) & 1)) {
                    atomicExch(error_flag, 30);
                    *abort_flag = 1;
                    break;
                }
                tc_fence_after();
                const uint32_t vst = v_smem + sv * V_TILE;
#pragma unroll
                for (int kk = 0; kk < FA_KEYS / 16; kk++) {
                    const uint64_t dv = smem_desc_mn_sw128(vst + kk * 16 * 128, FA_HALF_BYTES, 1024);
                    umma_bf16_ts(tm_o, tmem_base + s * 128 + kk * 8, dv, idesc_pv, (it | kk) ? 1u : 0u);
                    umma_bf16_ts(tm_o, tmem_base + s * 128 + 64 + kk * 8, dv, idesc_pv, 1u);
                }
                umma_commit(v_empty0 + 8 * sv);               // the value tile is used up
                umma_commit(pv_done);
            }
        }
    } else if (n_it > 0) {
        // ---------------------------------------------------------------- softmax and output
        const int q = warp & 3, r = q * 32 + lane;            // query row of this thread = TMEM lane
        const int hf = (warp - 2) >> 2;                       // which 64 key columns (and which half of the output columns) of the row
        constexpr int OC = VDP / 2;                           // output columns per thread: 32 or 64
        const uint32_t lane_base = (uint32_t)(q * 32) << 16;
        const int qpos = first_pos + r;
        const int lo = hb_oldest_visible(qpos, window, chunk);
        const bool valid = row_base + r < n_new;
        float m_run = -INFINITY, l = 0.0f;                    // l: this thread's columns only
        bool ok = true;
        for (int it = 0; it < n_it; it++) {
            const int s = it & 1;
            if (!mbar_wait(s_full0 + 8 * s, (it >> 1) & 1)) {
                atomicExch(error_flag, 27);
                *abort_flag = 1;
            }
            tc_fence_after();
            const uint32_t tm_s = tmem_base + s * 128 + lane_base;
            const int kbase = (jt0 + it) * FA_KEYS + hf * 64;
            // this thread's row sees keys lo..qpos; as columns of its half tile: [c_lo, c_hi]
            const int c_lo = lo - kbase, c_hi = qpos - kbase;
            float sv[64];
            tmem_ld64(tm_s + hf * 64, sv);
            if (c_lo > 0 || c_hi < 63) {                       // the causal diagonal or the window's edge
#pragma unroll
                for (int e = 0; e < 64; e++)
                    if (e < c_lo || e > c_hi) sv[e] = -INFINITY;
            }
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int e = 0; e < 64; e += 4) {
                mx4[0] = fmaxf(mx4[0], sv[e]);
                mx4[1] = fmaxf(mx4[1], sv[e + 1]);
                mx4[2] = fmaxf(mx4[2], sv[e + 2]);
                mx4[3] = fmaxf(mx4[3], sv[e + 3]);
            }
            xrow[hf * 128 + r] = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
            // all 256 softmax threads: every score is in registers now (P may overwrite S) and the other half's maximum is
            // visible
            asm volatile("bar.sync 2, 256;" ::: "memory");
            if (*abort_flag) {                                 // read after the barrier: the same for all 256 threads
                ok = false;
                break;
            }
            const float m_tile = fmaxf(xrow[r], xrow[128 + r]) * scale_log2e;
            if (it == 0) {
                m_run = m_tile;
                if (sink != nullptr) {
                    // one more term exp(sink) of the row's sum, with no value: counted by one of the row's two threads
                    const float t0 = sink[head] * FA_LOG2E;
                    m_run = fmaxf(m_tile, t0);
                    if (hf == 0) l = exp2f(t0 - m_run);
                }
            } else {
                const bool grow = m_tile > m_run + FA_RESCALE_THRESHOLD;
                if (__any_sync(0xffffffffu, grow)) {
                    // the accumulator may only be touched between two of its MMAs
                    if (!mbar_wait(pv_done, (it - 1) & 1)) {
                        atomicExch(error_flag, 28);
                        *abort_flag = 1;
                    }
                    tc_fence_after();
                    const float m_new = fmaxf(m_run, m_tile);
                    const float corr = m_new == -INFINITY ? 1.0f : exp2f(m_run - m_new);
                    m_run = m_new;
                    l *= corr;
#pragma unroll 1
                    for (int c = 0; c < OC / 32; c++) {
                        float v[32];
                        tmem_ld32(tm_o + lane_base + hf * OC + c * 32, v);
#pragma unroll
                        for (int e = 0; e < 32; e++) v[e] *= corr;
                        tmem_st32(tm_o + lane_base + hf * OC + c * 32, v);
                    }
                    tmem_wait_st();
                }
            }
            const float neg_m = m_run == -INFINITY ? 0.0f : -m_run;
            float sum2[2] = {0.0f, 0.0f};
#pragma unroll
            for (int c = 0; c < 2; c++) {
                uint32_t hi[16], lo_t[16];
#pragma unroll
                for (int e = 0; e < 32; e += 2) {
                    const float p0 = exp2_approx(fmaf(sv[c * 32 + e], scale_log2e, neg_m));
                    const float p1 = exp2_approx(fmaf(sv[c * 32 + e + 1], scale_log2e, neg_m));
                    sum2[0] += p0;
                    sum2[1] += p1;
                    const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
                    const float2 hf2 = __bfloat1622float2(h);
                    hi[e >> 1] = *reinterpret_cast<const uint32_t*>(&h);
                    lo_t[e >> 1] = pack_bf16_pair(p0 - hf2.x, p1 - hf2.y);
                }
                tmem_st16u(tm_s + hf * 32 + c * 16, hi);      // P over S: the leading terms, then the rests
                tmem_st16u(tm_s + 64 + hf * 32 + c * 16, lo_t);
            }
            l += sum2[0] + sum2[1];
            tmem_wait_st();
            // The wait for the last product, behind the loop, tells phases apart by their parity: the product before it must be
            // done by then.  (Inside the loop it is: S_it is complete only after every product issued before it.)
            if (it + 1 == n_it && it > 0 && !mbar_wait(pv_done, (it - 1) & 1)) {
                atomicExch(error_flag, 28);
                *abort_flag = 1;
            }
            tc_fence_before();
            mbar_arrive(p_full0 + 8 * s);
        }
        // the row's gates, while the last product runs: 1 / (1 + exp(-g)) of this thread's output columns
        const int t = t_begin + row_base + r;
        const float* gr = gate != nullptr && valid ? gate + (size_t)t * ldg : nullptr;
        const bool each = gr != nullptr && gate_per > 1;
        float gv[OC];
#pragma unroll
        for (int c = 0; c < OC; c++) gv[c] = 1.0f;
        if (each) {
            const float* ge = gr + (size_t)head * vd + hf * OC;
            if (((uintptr_t)ge & 15) == 0) {
#pragma unroll
                for (int c = 0; c < OC; c += 4)
                    if (hf * OC + c < vd) {                    // (vd is a multiple of 8)
                        const float4 g4 = *reinterpret_cast<const float4*>(ge + c);
                        gv[c] = g4.x;
                        gv[c + 1] = g4.y;
                        gv[c + 2] = g4.z;
                        gv[c + 3] = g4.w;
                    }
            } else {
#pragma unroll
                for (int c = 0; c < OC; c++)
                    if (hf * OC + c < vd) gv[c] = ge[c];
            }
#pragma unroll
            for (int c = 0; c < OC; c++) gv[c] = 1.0f / (1.0f + expf(-gv[c]));
        }
        if (ok && !mbar_wait(pv_done, (n_it - 1) & 1)) {
            atomicExch(error_flag, 29);
            *abort_flag = 1;
        }
        // the two halves of a row add their sums
        asm volatile("bar.sync 2, 256;" ::: "memory");      // nobody still reads the maxima
        xrow[hf * 128 + r] = l;
        asm volatile("bar.sync 2, 256;" ::: "memory");
        if (!*abort_flag) {
            tc_fence_after();
            const float lt = xrow[r] + xrow[128 + r];
            float inv = lt > 0.0f ? 1.0f / lt : 0.0f;
            if (gr != nullptr && gate_per == 1) inv *= 1.0f / (1.0f + expf(-gr[head]));
            bf16* dst = out + (size_t)t * out_stride + (size_t)head * vd;
#pragma unroll
            for (int c = 0; c < OC / 32; c++) {
                const int col = hf * OC + c * 32;
                float v[32];
                tmem_ld32(tm_o + lane_base + col, v);          // (the whole warp)
                if (valid) {
#pragma unroll
                    for (int e = 0; e < 32; e += 8) {
                        if (col + e >= vd) break;
                        float w[8];
#pragma unroll
                        for (int k = 0; k < 8; k++) w[k] = v[e + k] * inv * gv[c * 32 + e + k];
                        uint4 o4;
                        o4.x = pack_bf16_pair(w[0], w[1]);
                        o4.y = pack_bf16_pair(w[2], w[3]);
                        o4.z = pack_bf16_pair(w[4], w[5]);
                        o4.w = pack_bf16_pair(w[6], w[7]);
                        *reinterpret_cast<uint4*>(dst + col + e) = o4;
                    }
                }
            }
            if (ones > 0 && head == 0 && hf == 0 && valid)
                for (int e = 0; e < ones; e++) dst[(size_t)nh * vd + e] = __float2bfloat16_rn(e == 0 ? 1.0f : 0.0f);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, 512);
    }
}

extern "C" int hb_attention_sink_prefill_tc_supported(int n_heads, int n_kv_heads, int head_dim, int v_dim) {
    return head_dim > 0 && head_dim <= 192 && head_dim % 8 == 0 && v_dim > 0 && v_dim <= 128 && v_dim % 8 == 0 && n_kv_heads > 0
           && n_heads % n_kv_heads == 0;
}

template <int HDP, int VDP>
static int launch_sink_tc(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const int* page_table, int pt_width,
                          const int* seq_start, const int* seq_pos0, void* out, long long out_stride, int ones, const float* gate, long long ldg,
                          int gate_per, int n_seqs, int q_blocks, int nh, int nkv, int hd, int vd, float scale, int window, int chunk,
                          const float* sink, int n_pages, int* error_flag, cudaStream_t stream) {
    constexpr int K_TILE = HDP / 64 * FA_HALF_BYTES, V_TILE = VDP / 64 * FA_HALF_BYTES;
    constexpr int SMEM = K_TILE + st_stages<HDP>::N * (K_TILE + V_TILE) + 18 * 8 + 16 + 2 * 128 * 4 + 1024;
    static_assert(SMEM <= 227 * 1024, "attention tiles do not fit shared memory");
    static_assert(st_stages<HDP>::N <= 3, "the barriers are laid out for three stages at most");
    static bool attr_done[HB_MAX_DEVICES] = {};
    bool& attr_set = attr_done[hb_device_slot()];
    if (!attr_set) {
        cudaError_t e = cudaFuncSetAttribute(attn_sink_prefill_tc_kernel<HDP, VDP>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (e != cudaSuccess) return hb_fail("attention_sink_prefill_tc: cannot reserve %d bytes of shared memory: %s", SMEM, cudaGetErrorString(e));
        attr_set = true;
    }
    cudaError_t e = hb_launch(attn_sink_prefill_tc_kernel<HDP, VDP>, dim3(nh, q_blocks), dim3(FA_THREADS), SMEM, stream, mq, mk, mv, page_table,
                              pt_width, seq_start, seq_pos0, (bf16*)out, out_stride, ones, gate, ldg, gate_per, n_seqs, nh, nkv, hd, vd,
                              scale * FA_LOG2E, window, chunk, sink, n_pages, error_flag);
    if (e != cudaSuccess) return hb_fail("attention_sink_prefill_tc: launch failed: %s", cudaGetErrorString(e));
    return hb_check_launch("attention_sink_prefill_tc");
}

// q: [tokens, q_stride] (head j at columns [j*hd, (j+1)*hd)); caches [n_pages][n_kv_heads][64][hd | vd]; out [tokens, out_stride]
// bfloat16: head j's results at columns [j*vd, (j+1)*vd), times sigmoid(gate) (gate_per 1: gate[t][head]; v_dim: gate[t][head * vd +
// d]; null: none), then `ones` columns of a one and zeros; q_blocks = sum over sequences of ceil(new tokens / 128).
extern "C" int hb_attention_sink_prefill_tc(const void* q, long long q_stride, long long n_tokens, const void* k_cache, const void* v_cache,
                                            const int* page_table, int pt_width, const int* seq_start, const int* seq_pos0, void* out,
                                            long long out_stride, int ones, const float* gate, long long ldg, int gate_per, int n_seqs,
                                            int q_blocks, int n_heads, int n_kv_heads, int head_dim, int v_dim, float scale, int window,
                                            int chunk, const float* sink, int n_pages, int* error_flag, void* stream) {
    if (n_seqs == 0 || q_blocks == 0) return 0;
    HB_REQUIRE(hb_attention_sink_prefill_tc_supported(n_heads, n_kv_heads, head_dim, v_dim),
               "attention_sink_prefill_tc: head sizes %d and %d are not built (multiples of 8, keys up to 192, values up to 128)", head_dim, v_dim);
    HB_REQUIRE(n_tokens > 0 && n_pages > 0 && q_blocks <= 65535 && error_flag != nullptr && window >= 0 && chunk >= 0 && ones >= 0,
               "attention_sink_prefill_tc: bad sizes");
    HB_REQUIRE(chunk == 0 || window == 0, "attention_sink_prefill_tc: chunks come without a window");
    HB_REQUIRE(q_stride % 8 == 0 && ((uintptr_t)q & 15) == 0, "attention_sink_prefill_tc: queries must have 16-byte aligned rows");
    HB_REQUIRE(out_stride % 8 == 0 && ((uintptr_t)out & 15) == 0 && out_stride >= (long long)n_heads * v_dim + ones,
               "attention_sink_prefill_tc: output must have 16-byte aligned rows that hold the heads");
    HB_REQUIRE(((uintptr_t)k_cache & 15) == 0 && ((uintptr_t)v_cache & 15) == 0, "attention_sink_prefill_tc: cache must be 16-byte aligned");
    HB_REQUIRE(gate == nullptr || ((gate_per == 1 || gate_per == v_dim) && ldg >= (long long)n_heads * gate_per),
               "attention_sink_prefill_tc: a gate per (token, head) or per element expected");
    CUtensorMap mq, mk, mv;
    const long long cache_rows = (long long)n_pages * n_kv_heads * HB_PAGE_TOKENS;
    if (tc_make_map(&mq, q, n_tokens, (long long)n_heads * head_dim, q_stride, FA_ROWS)) return 1;
    if (tc_make_map(&mk, k_cache, cache_rows, head_dim, head_dim, HB_PAGE_TOKENS)) return 1;
    if (tc_make_map(&mv, v_cache, cache_rows, v_dim, v_dim, HB_PAGE_TOKENS)) return 1;
    cudaStream_t st = (cudaStream_t)stream;
#define HB_ST(HDP, VDP)                                                                                                                    \
    return launch_sink_tc<HDP, VDP>(mq, mk, mv, page_table, pt_width, seq_start, seq_pos0, out, out_stride, ones, gate, ldg, gate_per, n_seqs, \
                                    q_blocks, n_heads, n_kv_heads, head_dim, v_dim, scale, window, chunk, sink, n_pages, error_flag, st)
    if (v_dim <= 64) {
        if (head_dim <= 64) HB_ST(64, 64);
        if (head_dim <= 128) HB_ST(128, 64);
        HB_ST(192, 64);
    }
    if (head_dim <= 64) HB_ST(64, 128);
    if (head_dim <= 128) HB_ST(128, 128);
    HB_ST(192, 128);
#undef HB_ST
}
