// Group-wise RMS norms: with `groups` = G and n values a row, value i of run r = i / (n / G) becomes
// x_i / sqrt((G / n) sum_{j in run r} x_j^2 + eps) * w_i (G = 1: the ordinary RMS norm).
//
// group_rmsnorm:   out[i] = norm(x[rows[i]])  (rows null: every row), in the dtype the next product reads.
// gated_sum_norm:  x[t] = norm(alpha * x[t] + sigmoid(g[t] + b) * sum_k y[t * n_sum + k]): a sublayer's result on its way
//                  into the 32-bit residual stream when the norm sits behind the sum.  The gate's logits g and bias b may be
//                  absent (the result then enters as it is); a sublayer may leave its result in n_sum rows per token that
//                  add up to it (the experts of a mixture), which this kernel sums in their order.  With `copy` the new row
//                  of x is also written there in copy's dtype: the sublayers of such a block read the stream itself, and a
//                  bfloat16 product reads this copy.
// Everything in 32-bit.  One block per token; the block's eight warps are dealt out to the groups (several warps to a group
// when there are fewer than eight groups, several groups to a warp when there are more), so a group's sum needs the warps of
// its own team only; a thread keeps its values in registers between the sum and the scaling.
#include "api.h"
#include "common.cuh"

#define GN_THREADS 256
#define GN_WARPS (GN_THREADS / 32)
// KEEP: vectors of VEC values a thread keeps in registers between the two (2 or 4, by the run's length: fewer registers, more
// blocks on an SM); what lies behind them is read again.

template <int VEC> struct gn_vec { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ gn_vec<VEC> gn_load(const float* p) {
    gn_vec<VEC> r;
    if (VEC == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        r.v[0] = q.x;
        r.v[1 % VEC] = q.y;
        r.v[2 % VEC] = q.z;
        r.v[3 % VEC] = q.w;
    } else {
#pragma unroll
        for (int i = 0; i < VEC; i++) r.v[i] = p[i];
    }
    return r;
}

template <int VEC>
__device__ __forceinline__ void gn_store(float* p, const gn_vec<VEC>& r) {
    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % VEC], r.v[2 % VEC], r.v[3 % VEC]);
    else {
#pragma unroll
        for (int i = 0; i < VEC; i++) p[i] = r.v[i];
    }
}

template <int VEC>
__device__ __forceinline__ void gn_store(bf16* p, const gn_vec<VEC>& r) {
    if (VEC == 4) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1 % VEC]), hi = __floats2bfloat162_rn(r.v[2 % VEC], r.v[3 % VEC]);
        uint2 pk;
        pk.x = *reinterpret_cast<uint32_t*>(&lo);
        pk.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = pk;
    } else {
#pragma unroll
        for (int i = 0; i < VEC; i++) p[i] = from_f32<bf16>(r.v[i]);
    }
}

// `load(i)` gives the row's values i .. i + VEC - 1 (it may be called twice for one i, always before that i is stored by the
// same thread), `store(i, values)` takes the normed and weighted ones.
template <int VEC, int KEEP, typename Load, typename Store>
__device__ __forceinline__ void gn_row(int n, int groups, float eps, const float* __restrict__ w, float* scratch, Load load, Store store) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int size = n / groups;
    const int wpg = groups >= GN_WARPS ? 1 : GN_WARPS / groups;         // warps of a team
    const int teams = GN_WARPS / wpg, team = warp / wpg, sub = warp - team * wpg;
    const int first = (sub * 32 + lane) * VEC, stride = wpg * 32 * VEC;
    const int rounds = (groups + teams - 1) / teams;                    // one whenever a team has several warps
    for (int it = 0; it < rounds; it++) {
        const int g = team + it * teams;
        const bool on = team < teams && g < groups;
        const int base = g * size;
        gn_vec<VEC> keep[KEEP];
        float ss = 0.0f;
#pragma unroll
        for (int s = 0; s < KEEP; s++) {
            const int i = first + s * stride;
            if (on && i < size) {
                keep[s] = load(base + i);
#pragma unroll
                for (int k = 0; k < VEC; k++) ss = fmaf(keep[s].v[k], keep[s].v[k], ss);
            }
        }
        for (int i = first + KEEP * stride; on && i < size; i += stride) {
            const gn_vec<VEC> v = load(base + i);
#pragma unroll
            for (int k = 0; k < VEC; k++) ss = fmaf(v.v[k], v.v[k], ss);
        }
        ss = warp_sum(ss);
        if (wpg > 1) {
            if (lane == 0) scratch[warp] = ss;
            __syncthreads();
            ss = 0.0f;
            if (on)
                for (int j = 0; j < wpg; j++) ss += scratch[team * wpg + j];
        }
        const float r = 1.0f / sqrtf(ss / (float)size + eps);
#pragma unroll
        for (int s = 0; s < KEEP; s++) {
            const int i = first + s * stride;
            if (on && i < size) {
                const gn_vec<VEC> ww = gn_load<VEC>(w + base + i);
#pragma unroll
                for (int k = 0; k < VEC; k++) keep[s].v[k] = keep[s].v[k] * r * ww.v[k];
                store(base + i, keep[s]);
            }
        }
        for (int i = first + KEEP * stride; on && i < size; i += stride) {
            gn_vec<VEC> v = load(base + i);
            const gn_vec<VEC> ww = gn_load<VEC>(w + base + i);
#pragma unroll
            for (int k = 0; k < VEC; k++) v.v[k] = v.v[k] * r * ww.v[k];
            store(base + i, v);
        }
    }
}

template <typename TO, int VEC, int KEEP>
__global__ void __launch_bounds__(GN_THREADS)
group_rmsnorm_kernel(const float* __restrict__ x, long long ldx, const float* __restrict__ w, float eps, int groups, TO* __restrict__ out,
                     long long ldo, const int* __restrict__ rows, int n) {
    pdl_trigger();
    __shared__ float scratch[GN_WARPS];
    pdl_wait();
    x = pdl_fresh(x);
    const int t = blockIdx.x;
    const float* xr = x + (size_t)(rows ? rows[t] : t) * ldx;
    TO* o = out + (size_t)t * ldo;
    gn_row<VEC, KEEP>(n, groups, eps, w, scratch, [&](int i) { return gn_load<VEC>(xr + i); }, [&](int i, const gn_vec<VEC>& v) { gn_store<VEC>(o + i, v); });
}

template <typename TC, int VEC, int KEEP>
__global__ void __launch_bounds__(GN_THREADS, KEEP == 2 ? 5 : 4)
gated_sum_norm_kernel(float* __restrict__ x, long long ldx, float alpha, const float* __restrict__ y, long long ldy, int n_sum,
                      const float* __restrict__ gate, long long ldg, const float* __restrict__ gate_bias, const float* __restrict__ w,
                      float eps, int groups, TC* __restrict__ copy, long long ldc, int n) {
    pdl_trigger();
    __shared__ float scratch[GN_WARPS];
    pdl_wait();
    x = pdl_fresh(x);
    y = pdl_fresh(y);
    gate = pdl_fresh(gate);
    const int t = blockIdx.x;
    float* xr = x + (size_t)t * ldx;
    const float* yr = y + (size_t)t * n_sum * ldy;
    const float* gr = gate ? gate + (size_t)t * ldg : nullptr;
    auto load = [&](int i) {
        gn_vec<VEC> v = gn_load<VEC>(yr + i);
        for (int j = 1; j < n_sum; j++) {
            const gn_vec<VEC> u = gn_load<VEC>(yr + (size_t)j * ldy + i);
#pragma unroll
            for (int k = 0; k < VEC; k++) v.v[k] += u.v[k];
        }
        if (gr != nullptr) {
            gn_vec<VEC> g = gn_load<VEC>(gr + i);
            if (gate_bias != nullptr) {
                const gn_vec<VEC> b = gn_load<VEC>(gate_bias + i);
#pragma unroll
                for (int k = 0; k < VEC; k++) g.v[k] += b.v[k];
            }
#pragma unroll
            for (int k = 0; k < VEC; k++) v.v[k] *= 1.0f / (1.0f + expf(-g.v[k]));
        }
        const gn_vec<VEC> a = gn_load<VEC>(xr + i);
#pragma unroll
        for (int k = 0; k < VEC; k++) v.v[k] = fmaf(alpha, a.v[k], v.v[k]);
        return v;
    };
    auto store = [&](int i, const gn_vec<VEC>& v) {
        gn_store<VEC>(xr + i, v);
        if (copy != nullptr) gn_store<VEC>(copy + (size_t)t * ldc + i, v);
    };
    gn_row<VEC, KEEP>(n, groups, eps, w, scratch, load, store);
}

// whether two vectors a thread hold a whole run
static bool gn_short(int n, int groups, int vec) {
    const int wpg = groups >= GN_WARPS ? 1 : GN_WARPS / groups;
    return n / groups <= 2 * wpg * 32 * vec;
}

static bool gn_aligned(const void* p, long long ld, int elem) { return ((uintptr_t)p & (elem * 4 - 1)) == 0 && ld % 4 == 0; }

extern "C" int hb_group_rmsnorm(const float* x, long long ldx, const float* w, float eps, int groups, void* out, int out_dtype,
                                long long ldo, const int* rows, int n_rows, int n, void* stream) {
    if (n_rows == 0) return 0;
    HB_REQUIRE(n_rows > 0 && n > 0 && ldx >= n && ldo >= n, "group_rmsnorm: bad sizes");
    HB_REQUIRE(groups > 0 && n % groups == 0, "group_rmsnorm: %d groups do not divide a row of %d", groups, n);
    HB_REQUIRE(out_dtype == HB_BF16 || out_dtype == HB_F32, "group_rmsnorm: unsupported output dtype %d", out_dtype);
    const bool vec = (n / groups) % 4 == 0 && gn_aligned(x, ldx, 4) && gn_aligned(w, 4, 4) && gn_aligned(out, ldo, out_dtype == HB_BF16 ? 2 : 4);
    cudaStream_t s = (cudaStream_t)stream;
#define HB_GN_K(TO, V, K) hb_launch(group_rmsnorm_kernel<TO, V, K>, dim3(n_rows), dim3(GN_THREADS), 0, s, x, ldx, w, eps, groups, (TO*)out, ldo, rows, n)
#define HB_GN(TO, V) do { if (gn_short(n, groups, V)) HB_GN_K(TO, V, 2); else HB_GN_K(TO, V, 4); } while (0)
    if (out_dtype == HB_BF16) { if (vec) HB_GN(bf16, 4); else HB_GN(bf16, 1); }
    else { if (vec) HB_GN(float, 4); else HB_GN(float, 1); }
#undef HB_GN
#undef HB_GN_K
    return hb_check_launch("group_rmsnorm");
}

extern "C" int hb_gated_sum_norm(float* x, long long ldx, float alpha, const float* y, long long ldy, int n_sum, const float* gate, long long ldg,
                                 const float* gate_bias, const float* w, float eps, int groups, void* copy, int copy_dtype, long long ldc,
                                 int n_rows, int n, void* stream) {
    if (n_rows == 0) return 0;
    HB_REQUIRE(n_rows > 0 && n > 0 && ldx >= n && ldy >= n && n_sum >= 1 && (gate == nullptr || ldg >= n) && (copy == nullptr || ldc >= n),
               "gated_sum_norm: bad sizes");
    HB_REQUIRE(groups > 0 && n % groups == 0, "gated_sum_norm: %d groups do not divide a row of %d", groups, n);
    HB_REQUIRE(copy == nullptr || copy_dtype == HB_BF16 || copy_dtype == HB_F32, "gated_sum_norm: unsupported copy dtype %d", copy_dtype);
    const bool vec = (n / groups) % 4 == 0 && gn_aligned(x, ldx, 4) && gn_aligned(y, ldy, 4) && gn_aligned(w, 4, 4) &&
                     (gate == nullptr || gn_aligned(gate, ldg, 4)) && gn_aligned(gate_bias, 4, 4) &&
                     (copy == nullptr || gn_aligned(copy, ldc, copy_dtype == HB_BF16 ? 2 : 4));
    cudaStream_t s = (cudaStream_t)stream;
#define HB_GS_K(TC, V, K)                                                                                                               \
    hb_launch(gated_sum_norm_kernel<TC, V, K>, dim3(n_rows), dim3(GN_THREADS), 0, s, x, ldx, alpha, y, ldy, n_sum, gate, ldg, gate_bias, w, eps, \
              groups, (TC*)copy, ldc, n)
#define HB_GS(TC, V) do { if (gn_short(n, groups, V)) HB_GS_K(TC, V, 2); else HB_GS_K(TC, V, 4); } while (0)
    if (copy != nullptr && copy_dtype == HB_BF16) { if (vec) HB_GS(bf16, 4); else HB_GS(bf16, 1); }
    else { if (vec) HB_GS(float, 4); else HB_GS(float, 1); }
#undef HB_GS
#undef HB_GS_K
    return hb_check_launch("gated_sum_norm");
}
