// The sum behind two sublayers that stand side by side, with the norm of the next reader in the same pass:
//   x[t] += a * y[t] + b * (z[t] + sum_k w[t][k] r[t * n + k]) + v ;  out[t] = x[t] / sqrt(mean(x[t]^2) + eps) * (offset + nw)
// with a factor per channel (a, b) on each result.  y: the one sublayer's result; z: the other's, and / or its n rows per token
// r with a weight each (the chosen experts' results of a mixture, w null: weights of one); v: one vector for every token (what a
// pass over a run of layers adds in front of its first layer).  Every one of them may be absent (null), and so may the norm.
// Everything in 32-bit.  One block per token; a thread keeps its values of the new row in registers between the sum of squares
// and the scaling.
#include "api.h"
#include "common.cuh"

#define PS_THREADS 256

template <int VEC> struct ps_vec { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ ps_vec<VEC> ps_load(const float* p) {
    ps_vec<VEC> r;
    if constexpr (VEC == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    } else {
        r.v[0] = p[0];
    }
    return r;
}

template <int VEC>
__device__ __forceinline__ void ps_store(float* p, const ps_vec<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else p[0] = r.v[0];
}

template <int VEC>
__device__ __forceinline__ void ps_store(bf16* p, const ps_vec<VEC>& r) {
    if constexpr (VEC == 4) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 pk;
        pk.x = *reinterpret_cast<uint32_t*>(&lo);
        pk.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = pk;
    } else {
        p[0] = from_f32<bf16>(r.v[0]);
    }
}

// KEEP vectors of VEC values a thread stay in registers; what lies behind them (very wide rows) is read again.
template <typename TO, int VEC, int KEEP>
__global__ void __launch_bounds__(PS_THREADS)
parallel_sum_kernel(float* __restrict__ x, long long ldx, const float* __restrict__ y, long long ldy, const float* __restrict__ a,
                    const float* __restrict__ z, long long ldz, const float* __restrict__ r, long long ldr, const float* __restrict__ w, int n_rows_per,
                    const float* __restrict__ b, const float* __restrict__ v, const float* __restrict__ nw, float eps, float offset,
                    TO* __restrict__ out, long long ldo, int n) {
    pdl_trigger();
    __shared__ float scratch[33];
    pdl_wait();
    x = pdl_fresh(x);
    y = pdl_fresh(y);
    z = pdl_fresh(z);
    r = pdl_fresh(r);
    w = pdl_fresh(w);
    const int t = blockIdx.x;
    float* xr = x + (size_t)t * ldx;
    const float* wt = w ? w + (size_t)t * n_rows_per : nullptr;
    auto row_value = [&](int i) {
        ps_vec<VEC> s = ps_load<VEC>(xr + i);
        if (y != nullptr) {
            const ps_vec<VEC> yv = ps_load<VEC>(y + (size_t)t * ldy + i), av = ps_load<VEC>(a + i);
#pragma unroll
            for (int k = 0; k < VEC; k++) s.v[k] = fmaf(av.v[k], yv.v[k], s.v[k]);
        }
        if (b != nullptr) {
            ps_vec<VEC> f;
            if (z != nullptr) f = ps_load<VEC>(z + (size_t)t * ldz + i);
            else {
#pragma unroll
                for (int k = 0; k < VEC; k++) f.v[k] = 0.0f;
            }
#pragma unroll 4
            for (int j = 0; j < n_rows_per; j++) {
                const ps_vec<VEC> e = ps_load<VEC>(r + ((size_t)t * n_rows_per + j) * ldr + i);
                const float we = wt ? wt[j] : 1.0f;
#pragma unroll
                for (int k = 0; k < VEC; k++) f.v[k] = fmaf(we, e.v[k], f.v[k]);
            }
            const ps_vec<VEC> bv = ps_load<VEC>(b + i);
#pragma unroll
            for (int k = 0; k < VEC; k++) s.v[k] = fmaf(bv.v[k], f.v[k], s.v[k]);
        }
        if (v != nullptr) {
            const ps_vec<VEC> vv = ps_load<VEC>(v + i);
#pragma unroll
            for (int k = 0; k < VEC; k++) s.v[k] += vv.v[k];
        }
        ps_store<VEC>(xr + i, s);
        return s;
    };
    ps_vec<VEC> keep[KEEP];
    float ss = 0.0f;
    constexpr int STRIDE = PS_THREADS * VEC;
#pragma unroll
    for (int s = 0; s < KEEP; s++) {
        const int i = s * STRIDE + threadIdx.x * VEC;
        if (i < n) {
            keep[s] = row_value(i);
#pragma unroll
            for (int k = 0; k < VEC; k++) ss = fmaf(keep[s].v[k], keep[s].v[k], ss);
        }
    }
    for (int i = KEEP * STRIDE + threadIdx.x * VEC; i < n; i += STRIDE) {
        const ps_vec<VEC> s = row_value(i);
#pragma unroll
        for (int k = 0; k < VEC; k++) ss = fmaf(s.v[k], s.v[k], ss);
    }
    if (out == nullptr) return;
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
    TO* o = out + (size_t)t * ldo;
    auto emit = [&](int i, ps_vec<VEC> s) {
        const ps_vec<VEC> ww = ps_load<VEC>(nw + i);
#pragma unroll
        for (int k = 0; k < VEC; k++) s.v[k] = s.v[k] * inv * (offset + ww.v[k]);
        ps_store<VEC>(o + i, s);
    };
#pragma unroll
    for (int s = 0; s < KEEP; s++) {
        const int i = s * STRIDE + threadIdx.x * VEC;
        if (i < n) emit(i, keep[s]);
    }
    for (int i = KEEP * STRIDE + threadIdx.x * VEC; i < n; i += STRIDE) emit(i, ps_load<VEC>(xr + i));
}

static bool ps_aligned(const void* p, long long ld, int elem) { return ((uintptr_t)p & (elem * 4 - 1)) == 0 && ld % 4 == 0; }

// x [rows][n]; y, z [rows][n] or null; r [rows * n_sum][n] with weights w [rows][n_sum] (null: ones), n_sum 0: none; a (with y), b (with z or
// r), v, nw [n]; out [rows][n] or null.
extern "C" int hb_parallel_sum(float* x, long long ldx, const float* y, long long ldy, const float* a, const float* z, long long ldz, const float* r,
                               long long ldr, const float* w, int n_sum, const float* b, const float* v, const float* nw, float eps, float offset,
                               void* out, int out_dtype, long long ldo, int n_rows, int n, void* stream) {
    if (n_rows == 0) return 0;
    HB_REQUIRE(n_rows > 0 && n > 0 && ldx >= n && n_sum >= 0, "parallel_sum: bad sizes");
    HB_REQUIRE((y == nullptr || (a != nullptr && ldy >= n)) && (z == nullptr || ldz >= n) && (n_sum == 0 || (r != nullptr && ldr >= n)),
               "parallel_sum: a result without its factor, or rows that are too short");
    HB_REQUIRE((z != nullptr || n_sum > 0) == (b != nullptr), "parallel_sum: the second result and its factor come together");
    HB_REQUIRE(out == nullptr || (nw != nullptr && ldo >= n && (out_dtype == HB_BF16 || out_dtype == HB_F32)), "parallel_sum: bad norm output");
    const int oe = out_dtype == HB_BF16 ? 2 : 4;
    const bool vec = n % 4 == 0 && ps_aligned(x, ldx, 4) && (y == nullptr || ps_aligned(y, ldy, 4)) && (z == nullptr || ps_aligned(z, ldz, 4)) &&
                     (n_sum == 0 || ps_aligned(r, ldr, 4)) && ps_aligned(a, 4, 4) && ps_aligned(b, 4, 4) && ps_aligned(v, 4, 4) && ps_aligned(nw, 4, 4) &&
                     (out == nullptr || ps_aligned(out, ldo, oe));
    cudaStream_t s = (cudaStream_t)stream;
#define HB_PS_K(TO, V, K)                                                                                                                    \
    hb_launch(parallel_sum_kernel<TO, V, K>, dim3(n_rows), dim3(PS_THREADS), 0, s, x, ldx, y, ldy, a, z, ldz, r, ldr, w, n_sum, b, v, nw, eps, offset, \
              (TO*)out, ldo, n)
#define HB_PS(TO, V) do { if (n <= 2 * PS_THREADS * V) HB_PS_K(TO, V, 2); else HB_PS_K(TO, V, 4); } while (0)
    if (out != nullptr && out_dtype == HB_BF16) { if (vec) HB_PS(bf16, 4); else HB_PS(bf16, 1); }
    else { if (vec) HB_PS(float, 4); else HB_PS(float, 1); }
#undef HB_PS
#undef HB_PS_K
    return hb_check_launch("parallel_sum");
}
