// A token's own input to a layer: every token has, per layer, a vector of `dim` numbers in a table [vocab][ld] (layer i's at
// column i * dim); side_unit multiplies it by the tanh gelu of a product of the residual stream:
//   out[t][c] = gelu_tanh(s[t][c]) * E[token[t]][col0 + c]   for c < dim, 0 for the padding columns up to n_out,
// in the dtype the projection back to the model's width reads.  A warp per token for small vectors, everything in 32-bit.
#include "api.h"
#include "common.cuh"

#define TS_THREADS 128

template <typename TE, typename TO>
__global__ void __launch_bounds__(TS_THREADS)
side_unit_kernel(const float* __restrict__ s, long long lds, const int* __restrict__ tokens, const TE* __restrict__ table, long long ldt,
                 long long col0, int vocab, TO* __restrict__ out, long long ldo, int dim, int n_out, int n_tokens, int per_token, int* status) {
    pdl_trigger();
    pdl_wait();
    s = pdl_fresh(s);
    tokens = pdl_fresh(tokens);
    // per_token threads serve a token, TS_THREADS / per_token tokens a block
    const int t = blockIdx.x * (TS_THREADS / per_token) + threadIdx.x / per_token;
    if (t >= n_tokens) return;
    int tok = tokens[t];
    if (tok < 0 || tok >= vocab) {
        if (threadIdx.x % per_token == 0) hb_note(status, HB_STATUS_TOKEN, 1 + t);
        tok = 0;                           // never read outside the table
    }
    const float* sr = s + (size_t)t * lds;
    const TE* er = table + (size_t)tok * ldt + col0;
    TO* o = out + (size_t)t * ldo;
    for (int c = threadIdx.x % per_token; c < n_out; c += per_token) {
        float v = 0.0f;
        if (c < dim) {
            const float z = sr[c];
            v = 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))) * to_f32(er[c]);
        }
        o[c] = from_f32<TO>(v);
    }
}

extern "C" int hb_side_unit(const float* s, long long lds, const int* tokens, const void* table, int table_dtype, long long ldt, long long col0,
                            int vocab, void* out, int out_dtype, long long ldo, int dim, int n_out, int n_tokens, int* status, void* stream) {
    if (n_tokens == 0) return 0;
    HB_REQUIRE(n_tokens > 0 && dim > 0 && n_out >= dim && vocab > 0 && lds >= dim && ldo >= n_out && col0 >= 0 && ldt >= col0 + dim,
               "side_unit: bad sizes");
    const int per_token = dim <= 32 ? 32 : dim <= 64 ? 64 : 128, tokens_per_block = TS_THREADS / per_token;
    dim3 grid((n_tokens + tokens_per_block - 1) / tokens_per_block);
    cudaStream_t st = (cudaStream_t)stream;
#define HB_TS(TE, TO)                                                                                                                    \
    hb_launch(side_unit_kernel<TE, TO>, dim3(grid), dim3(TS_THREADS), 0, st, s, lds, tokens, (const TE*)table, ldt, col0, vocab, (TO*)out, ldo, dim, \
              n_out, n_tokens, per_token, status)
    if (table_dtype == HB_BF16 && out_dtype == HB_BF16) HB_TS(bf16, bf16);
    else if (table_dtype == HB_F32 && out_dtype == HB_F32) HB_TS(float, float);
    else if (table_dtype == HB_BF16 && out_dtype == HB_F32) HB_TS(bf16, float);
    else if (table_dtype == HB_F32 && out_dtype == HB_BF16) HB_TS(float, bf16);
    else return hb_fail("side_unit: unsupported dtypes %d -> %d", table_dtype, out_dtype);
#undef HB_TS
    return hb_check_launch("side_unit");
}
