// Softmax attention for steps of few tokens per sequence (decoding above all), one block per (token, key/value head, key range):
// the query heads of a group share the head's keys and values, so a cached row is read once for all of them, and no head's
// weights meet another head's values.  Causal, with a sliding window or chunks of positions, a sink, key and value heads of any
// size that is a multiple of 8, over the paged bfloat16 cache.  `v_in_k`: a value row is the first vd numbers of the key row
// (attention over cached latents), and only the key rows are read.
//
// Per page of 64 keys, brought in by a cp.async pipeline: scores of the group's query heads (the rows of 16-row mma.sync tiles, one
// or two) by warps that own 8 keys each; softmax bookkeeping by one warp per row, with the maximum and the sum in registers; the
// weighted values by warps that own 16-column tiles of the value head.  Scores, maximum, sum and accumulators are float32; the
// weights enter the second product as TWO bfloat16 terms, hi = bf16(p) and lo = bf16(p - hi), i.e. exact to 16 mantissa bits.
// One key range: the block writes the normalised result, times the gate (per head or per element), and the columns of ones
// behind the heads.  Several: unnormalised sums with (maximum, sum) go to scratch, and attention_group_combine adds them up.
#include "api.h"
#include "mma.cuh"

#define AG_THREADS 256
#define AG_WARPS 8
#define AG_KEYS HB_PAGE_TOKENS
// A row of scores (AG_KEYS floats) becomes a row of weights in its place: AG_KEYS leading terms, then AG_KEYS rests, bfloat16
#define AG_SST (AG_KEYS + 4)           // floats per row
#define AG_PST (2 * AG_SST)            // the same in bfloat16
#define AG_LOG2E 1.4426950408889634f
#define AG_SMEM_MAX (220 * 1024)
#define AG_MAX_SPLITS 64

struct AgSizes {
    int hd16, vd16, kst, vst, stages;
    size_t stage_elems, bytes;
};

static bool ag_sizes(int group, int hd, int vd, int v_in_k, AgSizes& z, int& mt) {
    mt = group > 16 ? 2 : 1;
    z.hd16 = (hd + 15) / 16 * 16;
    z.vd16 = (vd + 15) / 16 * 16;
    z.kst = z.hd16 + 8;
    z.vst = v_in_k ? z.kst : z.vd16 + 8;
    z.stage_elems = (size_t)AG_KEYS * (z.kst + (v_in_k ? 0 : z.vst));
    const size_t rows = 16 * (size_t)mt;
    const size_t fixed = rows * z.kst * 2 + rows * AG_SST * 4 + 2 * rows * 4;
    const size_t stage = z.stage_elems * 2;
    if (fixed + 2 * stage > AG_SMEM_MAX) return false;
    // two blocks on an SM where that leaves two stages, up to four stages
    const size_t two = 112 * 1024;
    z.stages = 2;
    while (z.stages < 4 && fixed + (z.stages + 1) * stage <= two) z.stages++;
    z.bytes = fixed + z.stages * stage;
    return true;
}

template <int MT, int PAIRS>
__global__ void __launch_bounds__(AG_THREADS)
attention_group_kernel(const bf16* __restrict__ q, long long ldq, const bf16* __restrict__ k_cache, const bf16* __restrict__ v_cache, int v_in_k,
                       const int* __restrict__ page_table, int pt_width, const int* __restrict__ tok_seq, const int* __restrict__ positions,
                       float* __restrict__ partial, float* __restrict__ ml, bf16* __restrict__ out_b, float* __restrict__ out_f, long long ldo,
                       int ones, const float* __restrict__ gate, long long ldg, int gate_per, int nh, int nkv, int chunks, int hd, int vd,
                       int hd16, int vd16, int kst, int vst, int stages, float scale_log2e, int window, int chunk_len,
                       const float* __restrict__ sink, int n_pages, int* status) {
    pdl_trigger();
    extern __shared__ __align__(128) unsigned char ag_smem[];
    constexpr int ROWS = 16 * MT;
    const int stage_elems = AG_KEYS * (kst + (v_in_k ? 0 : vst));
    bf16* stage0 = reinterpret_cast<bf16*>(ag_smem);
    bf16* Qs = stage0 + (size_t)stages * stage_elems;           // [ROWS][kst]
    float* Ss = reinterpret_cast<float*>(Qs + ROWS * kst);      // [ROWS][AG_SST]
    bf16* Ph = reinterpret_cast<bf16*>(Ss);                     // [ROWS][AG_PST]: leading terms, and AG_KEYS further on the rests
    bf16* Pl = Ph + AG_KEYS;
    float* c_s = Ss + ROWS * AG_SST;                            // [ROWS]: the accumulators' factor of this page
    float* l_s = c_s + ROWS;                                    // [ROWS]: the rows' sums, at the end

    const int split = blockIdx.x, splits = gridDim.x, t = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = blockIdx.y / chunks, group = nh / nkv;
    const int h0 = g * group + (blockIdx.y - g * chunks) * ROWS;              // first query head of this block
    const int rows = min(ROWS, (g + 1) * group - h0);
    const int p = positions[t];
    const int* pt = page_table + (size_t)tok_seq[t] * pt_width;
    const int lo = hb_oldest_visible(p, window, chunk_len);
    const int pg0 = lo / AG_KEYS, pg1 = p / AG_KEYS + 1, per = (pg1 - pg0 + splits - 1) / splits;
    const int p_begin = pg0 + split * per, n_it = max(0, min(pg1, p_begin + per) - p_begin);

    // what stays zero: the keys' and queries' columns behind the head (their products must vanish)
    if (hd16 > hd)
        for (int i = tid; i < stages * AG_KEYS; i += AG_THREADS) {
            bf16* row = stage0 + (size_t)(i / AG_KEYS) * stage_elems + (size_t)(i % AG_KEYS) * kst;
            for (int d = hd; d < hd16; d++) row[d] = __float2bfloat16_rn(0.0f);
        }
    if (tid < ROWS) c_s[tid] = 1.0f;

    pdl_wait();
    q = pdl_fresh(q);
    k_cache = pdl_fresh(k_cache);
    v_cache = pdl_fresh(v_cache);
    gate = pdl_fresh(gate);
    const int kc = hd / 8, vc = vd / 8;
    // a thread's 16-byte pieces of a page are AG_THREADS apart: the row and the piece of the row advance by fixed steps
    const int k_row0 = tid / kc, k_col0 = tid - k_row0 * kc, k_rows_on = AG_THREADS / kc, k_cols_on = AG_THREADS - k_rows_on * kc;
    const int v_row0 = tid / vc, v_col0 = tid - v_row0 * vc, v_rows_on = AG_THREADS / vc, v_cols_on = AG_THREADS - v_rows_on * vc;
    auto copy_rows = [&](uint32_t dst, const bf16* src, int per, int st, int r, int c, int rows_on, int cols_on) {
        const bf16* from = src + (size_t)tid * 8;
#pragma unroll 2
        while (r < AG_KEYS) {
            cp_async_16(dst + (uint32_t)(r * st + c * 8) * 2, from);
            from += AG_THREADS * 8;
            r += rows_on;
            c += cols_on;
            if (c >= per) {
                c -= per;
                r++;
            }
        }
    };
    bool bad_page = false;
    auto load_page = [&](int it) {
        if (it < n_it) {
            const int lp = p_begin + it;
            int page = lp < pt_width ? pt[lp] : -1;
            if (page < 0 || page >= n_pages) {                  // a fault of the host's bookkeeping: noted once, behind the loop
                bad_page = true;
                page = 0;
            }
            bf16* ks = stage0 + (size_t)(it % stages) * stage_elems;
            const bf16* ksrc = k_cache + ((size_t)page * nkv + g) * AG_KEYS * hd;
            const uint32_t kdst = (uint32_t)__cvta_generic_to_shared(ks);
            copy_rows(kdst, ksrc, kc, kst, k_row0, k_col0, k_rows_on, k_cols_on);
            if (!v_in_k)
                copy_rows(kdst + (uint32_t)(AG_KEYS * kst) * 2, v_cache + ((size_t)page * nkv + g) * AG_KEYS * vd, vc, vst, v_row0, v_col0, v_rows_on,
                          v_cols_on);
        }
        cp_async_commit();
    };
    for (int s = 0; s < stages - 1; s++) load_page(s);
    {
        const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
        const int qc = hd16 / 8;
        for (int i = tid; i < ROWS * qc; i += AG_THREADS) {
            const int r = i / qc, c = i - r * qc;
            *reinterpret_cast<uint4*>(Qs + r * kst + c * 8) =
                (r < rows && c < kc) ? *reinterpret_cast<const uint4*>(q + (size_t)t * ldq + (size_t)(h0 + r) * hd + c * 8) : zero;
        }
    }

    float acc[MT][PAIRS][2][4];
#pragma unroll
    for (int a = 0; a < MT; a++)
#pragma unroll
        for (int b = 0; b < PAIRS; b++)
#pragma unroll
            for (int c = 0; c < 2; c++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[a][b][c][e] = 0.0f;
    // the rows this warp keeps the books of: warp, warp + 8, ...; l is the lane's share of the sum
    float m_r[2 * MT], l_r[2 * MT];
#pragma unroll
    for (int i = 0; i < 2 * MT; i++) {
        const int row = warp + 8 * i;
        const bool with_sink = sink != nullptr && split == 0 && row < rows;    // a sink is where the first range starts
        m_r[i] = with_sink ? sink[h0 + row] * AG_LOG2E : -INFINITY;
        l_r[i] = with_sink && lane == 0 ? 1.0f : 0.0f;
    }
    const uint32_t q_base = (uint32_t)__cvta_generic_to_shared(Qs), ph_base = (uint32_t)__cvta_generic_to_shared(Ph);
    const uint32_t pl_base = ph_base + AG_KEYS * 2;
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8, r0 = lane >> 2;
    const int v_row = ((lane >> 3) & 1) * 8 + (lane & 7), v_chunk = lane >> 4;

    for (int it = 0; it < n_it; it++) {
        // this page's copies have landed (in the last turns the groups behind it are empty)
        if (stages == 2) cp_async_wait<0>();
        else if (stages == 3) cp_async_wait<1>();
        else cp_async_wait<2>();
        __syncthreads();
        load_page(it + stages - 1);
        const uint32_t kb = (uint32_t)__cvta_generic_to_shared(stage0 + (size_t)(it % stages) * stage_elems);
        const uint32_t vb = v_in_k ? kb : kb + (uint32_t)(AG_KEYS * kst) * 2;
        // scores of this warp's 8 keys
        {
            float s[MT][4];
#pragma unroll
            for (int a = 0; a < MT; a++) s[a][0] = s[a][1] = s[a][2] = s[a][3] = 0.0f;
            const uint32_t k_addr = kb + (uint32_t)((warp * 8 + (lane & 7)) * kst + (lane >> 3) * 8) * 2;
#pragma unroll 2
            for (int d0 = 0; d0 < hd16; d0 += 32) {
                uint32_t kf[4], qf[4];
                ldmatrix_x4(kf, k_addr + (uint32_t)d0 * 2);           // 32 columns; the second half may lie behind the row
#pragma unroll
                for (int a = 0; a < MT; a++) {
                    ldmatrix_x4(qf, q_base + (uint32_t)((a * 16 + a_row) * kst + d0 + a_col) * 2);
                    mma_bf16_16816(s[a], qf, kf[0], kf[1]);
                }
                if (d0 + 16 < hd16) {
#pragma unroll
                    for (int a = 0; a < MT; a++) {
                        ldmatrix_x4(qf, q_base + (uint32_t)((a * 16 + a_row) * kst + d0 + 16 + a_col) * 2);
                        mma_bf16_16816(s[a], qf, kf[2], kf[3]);
                    }
                }
            }
            const int c = warp * 8 + (lane & 3) * 2;
#pragma unroll
            for (int a = 0; a < MT; a++) {
                *reinterpret_cast<float2*>(Ss + (a * 16 + r0) * AG_SST + c) = make_float2(s[a][0], s[a][1]);
                *reinterpret_cast<float2*>(Ss + (a * 16 + r0 + 8) * AG_SST + c) = make_float2(s[a][2], s[a][3]);
            }
        }
        __syncthreads();
        const int key0 = (p_begin + it) * AG_KEYS + lane, key1 = key0 + 32;
#pragma unroll
        for (int i = 0; i < 2 * MT; i++) {
            const int row = warp + 8 * i;
            if (row >= rows) {                                      // (the same for the whole warp) no head owns this row: no weights
                const uint32_t none = 0u;
                *reinterpret_cast<uint32_t*>(Ph + row * AG_PST + 2 * lane) = none;
                *reinterpret_cast<uint32_t*>(Pl + row * AG_PST + 2 * lane) = none;
                continue;
            }
            const float s0 = (key0 >= lo && key0 <= p) ? Ss[row * AG_SST + lane] * scale_log2e : -INFINITY;
            const float s1 = (key1 >= lo && key1 <= p) ? Ss[row * AG_SST + lane + 32] * scale_log2e : -INFINITY;
            const float m_new = fmaxf(m_r[i], warp_max(fmaxf(s0, s1)));
            const float m_safe = m_new == -INFINITY ? 0.0f : m_new;
            const float corr = exp2f(m_r[i] - m_safe), p0 = exp2f(s0 - m_safe), p1 = exp2f(s1 - m_safe);
            m_r[i] = m_new;
            l_r[i] = l_r[i] * corr + p0 + p1;
            const bf16 hi0 = __float2bfloat16_rn(p0), hi1 = __float2bfloat16_rn(p1);
            __syncwarp();                                           // every lane has its scores: the weights may take their place
            Ph[row * AG_PST + lane] = hi0;
            Ph[row * AG_PST + lane + 32] = hi1;
            Pl[row * AG_PST + lane] = __float2bfloat16_rn(p0 - __bfloat162float(hi0));
            Pl[row * AG_PST + lane + 32] = __float2bfloat16_rn(p1 - __bfloat162float(hi1));
            if (lane == 0) c_s[row] = corr;
        }
        __syncthreads();
#pragma unroll
        for (int a = 0; a < MT; a++) {
            const float c0 = c_s[a * 16 + r0], c1 = c_s[a * 16 + r0 + 8];
#pragma unroll
            for (int b = 0; b < PAIRS; b++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    acc[a][b][c][0] *= c0;
                    acc[a][b][c][1] *= c0;
                    acc[a][b][c][2] *= c1;
                    acc[a][b][c][3] *= c1;
                }
        }
        // (small code: a block runs few pages, and what it has not yet run comes from L2)
#pragma unroll 1
        for (int ks = 0; ks < AG_KEYS / 16; ks++) {
            uint32_t ah[MT][4], al[MT][4];
#pragma unroll
            for (int a = 0; a < MT; a++) {
                const uint32_t off = (uint32_t)((a * 16 + a_row) * AG_PST + ks * 16 + a_col) * 2;
                ldmatrix_x4(ah[a], ph_base + off);
                ldmatrix_x4(al[a], pl_base + off);
            }
#pragma unroll
            for (int b = 0; b < PAIRS; b++) {
                const int c0 = (warp + AG_WARPS * b) * 16;
                if (c0 < vd16) {
                    uint32_t vf[4];
                    ldmatrix_x4_trans(vf, vb + (uint32_t)((ks * 16 + v_row) * vst + c0 + v_chunk * 8) * 2);
#pragma unroll
                    for (int a = 0; a < MT; a++) {
                        mma_bf16_16816(acc[a][b][0], ah[a], vf[0], vf[1]);
                        mma_bf16_16816(acc[a][b][0], al[a], vf[0], vf[1]);
                        mma_bf16_16816(acc[a][b][1], ah[a], vf[2], vf[3]);
                        mma_bf16_16816(acc[a][b][1], al[a], vf[2], vf[3]);
                    }
                }
            }
        }
    }
    cp_async_wait<0>();
    if (bad_page && tid == 0) hb_note(status, HB_STATUS_PAGE, 1 + tok_seq[t]);
    const bool whole = splits == 1;
#pragma unroll
    for (int i = 0; i < 2 * MT; i++) {
        const int row = warp + 8 * i;
        const float l = warp_sum(l_r[i]);
        if (lane == 0 && row < rows) {
            if (whole) l_s[row] = l;
            else *reinterpret_cast<float2*>(ml + (((size_t)t * nh + h0 + row) * splits + split) * 2) = make_float2(m_r[i], l);
        }
    }
    __syncthreads();
#pragma unroll
    for (int a = 0; a < MT; a++)
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int row = a * 16 + r0 + 8 * half;
            if (row >= rows) continue;
            const int h = h0 + row;
            float inv = 1.0f;
            if (whole) {
                inv = l_s[row] > 0.0f ? 1.0f / l_s[row] : 0.0f;
                if (gate != nullptr && gate_per == 1) inv *= 1.0f / (1.0f + expf(-gate[(size_t)t * ldg + h]));
            }
#pragma unroll
            for (int b = 0; b < PAIRS; b++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    const int d = (warp + AG_WARPS * b) * 16 + c * 8 + (lane & 3) * 2;
                    if (d >= vd) continue;                           // (vd is even: both columns of a pair are in or out)
                    float x = acc[a][b][c][2 * half] * inv, y = acc[a][b][c][2 * half + 1] * inv;
                    if (!whole) {
                        *reinterpret_cast<float2*>(partial + (((size_t)t * nh + h) * splits + split) * vd + d) = make_float2(x, y);
                        continue;
                    }
                    if (gate != nullptr && gate_per > 1) {
                        const float* ge = gate + (size_t)t * ldg + (size_t)h * vd + d;
                        x *= 1.0f / (1.0f + expf(-ge[0]));
                        y *= 1.0f / (1.0f + expf(-ge[1]));
                    }
                    const size_t o = (size_t)t * ldo + (size_t)h * vd + d;
                    if (out_f != nullptr) {
                        out_f[o] = x;
                        out_f[o + 1] = y;
                    } else {
                        out_b[o] = __float2bfloat16_rn(x);
                        out_b[o + 1] = __float2bfloat16_rn(y);
                    }
                }
        }
    if (whole && blockIdx.y == 0)
        for (int e = tid; e < ones; e += AG_THREADS) {
            const size_t o = (size_t)t * ldo + (size_t)nh * vd + e;
            if (out_f != nullptr) out_f[o] = e == 0 ? 1.0f : 0.0f;
            else out_b[o] = __float2bfloat16_rn(e == 0 ? 1.0f : 0.0f);
        }
}

// out[t, h*vd + d] = sum_s w_s partial[t, h, s, d] / sum_s w_s l_s with w_s = 2^(m_s - max m), times the gate; then the ones.
template <typename TO>
__global__ void __launch_bounds__(128)
attention_group_combine_kernel(const float* __restrict__ partial, const float* __restrict__ ml, TO* __restrict__ out, long long ldo, int nh,
                               int vd, int splits, int ones, const float* __restrict__ gate, long long ldg, int gate_per) {
    pdl_trigger();
    pdl_wait();
    partial = pdl_fresh(partial);
    ml = pdl_fresh(ml);
    gate = pdl_fresh(gate);
    __shared__ float ws[AG_MAX_SPLITS];
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const float* r = ml + ((size_t)t * nh + h) * splits * 2;
    if (tid < 32) {
        float M = -INFINITY, den = 0.0f;
        for (int s = tid; s < splits; s += 32) M = fmaxf(M, r[2 * s]);
        M = warp_max(M);
        for (int s = tid; s < splits; s += 32) {
            const float w = r[2 * s] == -INFINITY ? 0.0f : exp2f(r[2 * s] - M);
            ws[s] = w;
            den = fmaf(w, r[2 * s + 1], den);
        }
        den = warp_sum(den);
        float inv = den > 0.0f ? 1.0f / den : 0.0f;
        if (gate != nullptr && gate_per == 1) inv *= 1.0f / (1.0f + expf(-gate[(size_t)t * ldg + h]));
        for (int s = tid; s < splits; s += 32) ws[s] *= inv;
    }
    __syncthreads();
    const float* pr = partial + ((size_t)t * nh + h) * splits * vd;
    TO* o = out + (size_t)t * ldo + (size_t)h * vd;
    const float* ge = gate != nullptr && gate_per > 1 ? gate + (size_t)t * ldg + (size_t)h * vd : nullptr;
    // four columns a thread (vd is a multiple of 8), the ranges' rows eight loads at a time
    for (int d = tid * 4; d < vd; d += 128 * 4) {
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
        for (int s = 0; s < splits; s++) {
            const float w = ws[s];
            const float4 x = *reinterpret_cast<const float4*>(pr + (size_t)s * vd + d);
            v.x = fmaf(w, x.x, v.x);
            v.y = fmaf(w, x.y, v.y);
            v.z = fmaf(w, x.z, v.z);
            v.w = fmaf(w, x.w, v.w);
        }
        float r4[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int k = 0; k < 4; k++) {
            if (ge != nullptr) r4[k] *= 1.0f / (1.0f + expf(-ge[d + k]));
            o[d + k] = from_f32<TO>(r4[k]);
        }
    }
    if (h == 0)
        for (int e = tid; e < ones; e += 128) out[(size_t)t * ldo + (size_t)nh * vd + e] = from_f32<TO>(e == 0 ? 1.0f : 0.0f);
}

// The blocks of this kernel that one SM holds for these sizes, 0 when they are not built.
extern "C" int hb_attention_group_supported(int n_heads, int n_kv_heads, int head_dim, int v_dim, int v_in_k) {
    if (n_heads <= 0 || n_kv_heads <= 0 || n_heads % n_kv_heads || head_dim <= 0 || v_dim <= 0 || head_dim % 8 || v_dim % 8 || v_dim > 512) return 0;
    if (v_in_k && v_dim > head_dim) return 0;
    AgSizes z;
    int mt;
    if (!ag_sizes(n_heads / n_kv_heads, head_dim, v_dim, v_in_k, z, mt)) return 0;
    return z.bytes <= 112 * 1024 ? 2 : 1;
}

template <int MT, int PAIRS>
static int ag_launch(dim3 grid, const AgSizes& z, cudaStream_t s, const void* q, long long ldq, const void* kc, const void* vc, int v_in_k,
                     const int* page_table, int pt_width, const int* tok_seq, const int* positions, float* partial, float* ml, void* out,
                     int out_f32, long long ldo, int ones, const float* gate, long long ldg, int gate_per, int nh, int nkv, int chunks, int hd,
                     int vd, float scale, int window, int chunk, const float* sink, int n_pages, int* status) {
    static bool done[HB_MAX_DEVICES] = {};
    if (!done[hb_device_slot()]) {
        cudaError_t e = cudaFuncSetAttribute(attention_group_kernel<MT, PAIRS>, cudaFuncAttributeMaxDynamicSharedMemorySize, AG_SMEM_MAX);
        if (e != cudaSuccess) return hb_fail("attention_group: %s", cudaGetErrorString(e));
        done[hb_device_slot()] = true;
    }
    hb_launch(attention_group_kernel<MT, PAIRS>, dim3(grid), dim3(AG_THREADS), z.bytes, s, (const bf16*)q, ldq, (const bf16*)kc, (const bf16*)vc, v_in_k,
              page_table, pt_width, tok_seq, positions, partial, ml, out_f32 ? (bf16*)nullptr : (bf16*)out, out_f32 ? (float*)out : (float*)nullptr,
              ldo, ones, gate, ldg, gate_per, nh, nkv, chunks, hd, vd, z.hd16, z.vd16, z.kst, z.vst, z.stages, scale * AG_LOG2E, window, chunk,
              sink, n_pages, status);
    return hb_check_launch("attention_group");
}

// q [tokens, ldq] bfloat16; caches [n_pages][n_kv_heads][64][head_dim | v_dim] bfloat16 (v_in_k: v_cache is not read); out [tokens, ldo]
// bfloat16 or float32 (out_dtype).  splits > 1: scratch of tokens * heads * splits * (v_dim + 2) floats.
extern "C" int hb_attention_group(const void* q, long long ldq, const void* k_cache, const void* v_cache, int v_in_k, const int* page_table,
                                  int pt_width, const int* tok_seq, const int* positions, float* scratch, void* out, int out_dtype,
                                  long long ldo, int ones, const float* gate, long long ldg, int gate_per, int n_tokens, int n_heads,
                                  int n_kv_heads, int head_dim, int v_dim, float scale, int window, int chunk, const float* sink, int splits,
                                  int n_pages, int* status, void* stream) {
    if (n_tokens == 0) return 0;
    HB_REQUIRE(hb_attention_group_supported(n_heads, n_kv_heads, head_dim, v_dim, v_in_k) != 0, "attention_group: head sizes %d and %d are not built",
               head_dim, v_dim);
    HB_REQUIRE(n_tokens > 0 && n_tokens <= 65535 && splits >= 1 && splits <= AG_MAX_SPLITS && window >= 0 && chunk >= 0 && n_pages > 0 && ones >= 0,
               "attention_group: bad sizes");
    HB_REQUIRE(chunk == 0 || window == 0, "attention_group: chunks come without a window");
    HB_REQUIRE(splits == 1 || scratch != nullptr, "attention_group: no scratch for the key ranges");
    HB_REQUIRE(ldq % 8 == 0 && (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0, "attention_group: queries and cache must be 16-byte aligned");
    HB_REQUIRE(ldo >= (long long)n_heads * v_dim + ones && (out_dtype == HB_BF16 || out_dtype == HB_F32), "attention_group: bad output");
    HB_REQUIRE(gate == nullptr || ((gate_per == 1 || gate_per == v_dim) && ldg >= (long long)n_heads * gate_per),
               "attention_group: a gate per (token, head) or per element expected");
    AgSizes z;
    int mt;
    const int group = n_heads / n_kv_heads;
    ag_sizes(group, head_dim, v_dim, v_in_k, z, mt);
    const int chunks = (group + 16 * mt - 1) / (16 * mt);
    HB_REQUIRE((long long)n_kv_heads * chunks <= 65535 && n_heads <= 65535, "attention_group: too many heads");
    float* ml = scratch + (size_t)n_tokens * n_heads * splits * v_dim;
    dim3 grid(splits, n_kv_heads * chunks, n_tokens);
    cudaStream_t s = (cudaStream_t)stream;
    const int pairs = (z.vd16 / 16 + AG_WARPS - 1) / AG_WARPS;
    int rc;
#define HB_AG(MT, P)                                                                                                                        \
    rc = ag_launch<MT, P>(grid, z, s, q, ldq, k_cache, v_cache, v_in_k, page_table, pt_width, tok_seq, positions, scratch, ml, out,              \
                          out_dtype == HB_F32 ? 1 : 0, ldo, ones, gate, ldg, gate_per, n_heads, n_kv_heads, chunks, head_dim, v_dim, scale, window, \
                          chunk, sink, n_pages, status)
    if (mt == 1) { if (pairs <= 1) HB_AG(1, 1); else if (pairs <= 2) HB_AG(1, 2); else HB_AG(1, 4); }
    else { if (pairs <= 1) HB_AG(2, 1); else if (pairs <= 2) HB_AG(2, 2); else HB_AG(2, 4); }
#undef HB_AG
    if (rc || splits == 1) return rc;
    if (out_dtype == HB_BF16)
        hb_launch(attention_group_combine_kernel<bf16>, dim3(n_tokens, n_heads), dim3(128), 0, s, (const float*)scratch, (const float*)ml, (bf16*)out, ldo,
                  n_heads, v_dim, splits, ones, gate, ldg, gate_per);
    else
        hb_launch(attention_group_combine_kernel<float>, dim3(n_tokens, n_heads), dim3(128), 0, s, (const float*)scratch, (const float*)ml, (float*)out, ldo,
                  n_heads, v_dim, splits, ones, gate, ldg, gate_per);
    return hb_check_launch("attention_group_combine");
}
