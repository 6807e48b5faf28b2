// What a token brings to a layer by itself: a row of a table of its own, let through by a gate that
// reads the residual stream.
//
//     out[m, c] = gelu(z[m, c]) * table[token[m], column0 + c]       c in [0, dim)
//     gelu(z) = z / 2 * (1 + tanh(sqrt(2 / pi) * (z + 0.044715 z^3)))
//
// token_gate takes z as the product gave it.  token_gate_product computes z = W x as well, for steps of few
// rows: a block of eight warps takes one row and walks the outputs four at a time (16-byte pieces of the row
// and of four weight rows side by side, float32 sums over the warp by shuffles and over the warps in a fixed
// order), so that a row's result depends on nothing but the sizes.  With a pending pair of branch outputs the
// row is h + (s p + s' p'), rounded to the activation type: the block adds it up for itself and leaves h as
// it is (several blocks read it); whoever adds the token part to the stream adds the pair as well.
// A token outside the table sets THN_ERR_TOKEN_RANGE and reads row 0.
#include "common.cuh"

namespace {

__device__ __forceinline__ float gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
}

__device__ __forceinline__ int table_row(const int* tokens, int m, int n_table_rows, int* err) {
    const int token = tokens[m];
    if (token >= 0 && token < n_table_rows) return token;
    if (err) atomicOr(err, THN_ERR_TOKEN_RANGE);
    return 0;
}

template <typename T>
__global__ void __launch_bounds__(256) token_gate_kernel(T* __restrict__ out, const T* __restrict__ z,
                                                         const T* __restrict__ table, const int* __restrict__ tokens, int rows,
                                                         int dim, long long table_width, int column0, int n_table_rows,
                                                         int* __restrict__ err) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * dim) return;
    const int m = (int)(i / dim), c = (int)(i - (long long)m * dim);
    const int row = table_row(tokens, m, n_table_rows, err);
    out[i] = from_f32<T>(gelu_tanh(to_f32<T>(z[i])) * to_f32<T>(table[row * table_width + column0 + c]));
}

// The same, eight bfloat16 entries (16 bytes) per thread.
__global__ void __launch_bounds__(256) token_gate_bf16_vec_kernel(__nv_bfloat16* __restrict__ out,
                                                                  const __nv_bfloat16* __restrict__ z,
                                                                  const __nv_bfloat16* __restrict__ table,
                                                                  const int* __restrict__ tokens, int rows, int pieces,
                                                                  long long table_width, int column0, int n_table_rows,
                                                                  int* __restrict__ err) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * pieces) return;
    const int m = (int)(i / pieces), c = (int)(i - (long long)m * pieces);
    const uint4 zi = reinterpret_cast<const uint4*>(z)[i];
    const int row = table_row(tokens, m, n_table_rows, err);
    const uint4 ei = *reinterpret_cast<const uint4*>(table + row * table_width + column0 + c * 8);
    const __nv_bfloat162* z2 = reinterpret_cast<const __nv_bfloat162*>(&zi);
    const __nv_bfloat162* e2 = reinterpret_cast<const __nv_bfloat162*>(&ei);
    uint4 packed;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float2 v = __bfloat1622float2(z2[j]), e = __bfloat1622float2(e2[j]);
        o2[j] = __floats2bfloat162_rn(gelu_tanh(v.x) * e.x, gelu_tanh(v.y) * e.y);
    }
    reinterpret_cast<uint4*>(out)[i] = packed;
}

__device__ __forceinline__ float dot8(const uint4& a, const uint4& b, float acc) {
    const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&a);
    const __nv_bfloat162* y = reinterpret_cast<const __nv_bfloat162*>(&b);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 u = __bfloat1622float2(x[i]), v = __bfloat1622float2(y[i]);
        acc = fmaf(u.x, v.x, acc);
        acc = fmaf(u.y, v.y, acc);
    }
    return acc;
}

constexpr int kProductThreads = 256;

// The stream and the outputs that are still to be added to it (second may be null).
struct Pending {
    const float* h;
    const __nv_bfloat16 *first, *second;
    const float *scale1, *scale2;
};

__device__ __forceinline__ void eight(const float* p, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
__device__ __forceinline__ void eight(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const float2 f = __bfloat1622float2(pairs[k]);
        v[2 * k] = f.x, v[2 * k + 1] = f.y;
    }
}

template <bool PENDING>
__global__ void __launch_bounds__(kProductThreads) token_gate_product_kernel(
    __nv_bfloat16* __restrict__ out, const __nv_bfloat16* __restrict__ x, Pending pending, const __nv_bfloat16* __restrict__ w,
    const __nv_bfloat16* __restrict__ table, const int* __restrict__ tokens, int dim, int vecs, long long table_width,
    int column0, int n_table_rows, int* __restrict__ err) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ uint4 row[];          // PENDING: the row, rounded
    __shared__ float part[kProductThreads / 32][4];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, m = blockIdx.x;
    const uint4* a = PENDING ? row : reinterpret_cast<const uint4*>(x) + (size_t)m * vecs;
    if (PENDING) {
        const size_t base = (size_t)m * vecs * 8;
        for (int i = threadIdx.x; i < vecs; i += kProductThreads) {     // a thread reads back only what it wrote
            float v[8], s[8], p[8], f[8];
            eight(pending.h + base + i * 8, v);
            eight(pending.first + base + i * 8, s);
            eight(pending.scale1 + i * 8, f);
#pragma unroll
            for (int e = 0; e < 8; ++e) s[e] *= f[e];
            if (pending.second) {
                eight(pending.second + base + i * 8, p);
                eight(pending.scale2 + i * 8, f);
#pragma unroll
                for (int e = 0; e < 8; ++e) s[e] = fmaf(p[e], f[e], s[e]);
            }
            uint4 packed;
            __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
            for (int k = 0; k < 4; ++k)
                o2[k] = __floats2bfloat162_rn(__fadd_rn(v[2 * k], s[2 * k]), __fadd_rn(v[2 * k + 1], s[2 * k + 1]));
            row[i] = packed;
        }
    }
    const uint4* wv = reinterpret_cast<const uint4*>(w);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    for (int n0 = blockIdx.y * 4; n0 < dim; n0 += gridDim.y * 4) {
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (int i = threadIdx.x; i < vecs; i += kProductThreads) {
            uint4 b[4];
            const uint4 av = a[i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = n0 + j < dim ? __ldg(wv + (size_t)(n0 + j) * vecs + i) : zero;
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[j] = dot8(av, b[j], acc[j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float total = warp_sum(acc[j]);
            if (lane == 0) part[warp][j] = total;
        }
        __syncthreads();
        if (threadIdx.x < 4 && n0 + threadIdx.x < dim) {
            float z = 0.f;
#pragma unroll
            for (int k = 0; k < kProductThreads / 32; ++k) z += part[k][threadIdx.x];
            const int c = n0 + threadIdx.x, row = table_row(tokens, m, n_table_rows, err);
            out[(size_t)m * dim + c] =
                __float2bfloat16(gelu_tanh(z) * __bfloat162float(table[row * table_width + column0 + c]));
        }
        __syncthreads();
    }
}
}  // namespace

// z, out [rows, dim] of the activation type; table [n_table_rows, table_width] of the same type.
THN_API int thn_token_gate(void* out, const void* z, const void* table, const int* tokens, int rows, int dim, int table_width,
                           int column0, int n_table_rows, int dtype, int* err, cudaStream_t stream) {
    THN_CHECK_ARG(rows >= 0 && dim > 0 && column0 >= 0 && column0 + dim <= table_width && n_table_rows > 0,
                  "token_gate: columns [%d, %d) of a table of %d x %d", column0, column0 + dim, n_table_rows, table_width);
    if (rows == 0) return THN_OK;
    const bool vec = dtype == THN_BF16 && dim % 8 == 0 && table_width % 8 == 0 && column0 % 8 == 0 &&
                     (((uintptr_t)out | (uintptr_t)z | (uintptr_t)table) & 15) == 0;
    const long long items = (long long)rows * (vec ? dim / 8 : dim);
    const unsigned blocks = (unsigned)((items + 255) / 256);
    if (vec)
        thn_launch(token_gate_bf16_vec_kernel, blocks, 256, 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)z,
                   (const __nv_bfloat16*)table, tokens, rows, dim / 8, (long long)table_width, column0, n_table_rows, err);
    else if (dtype == THN_BF16)
        thn_launch(token_gate_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)z,
                   (const __nv_bfloat16*)table, tokens, rows, dim, (long long)table_width, column0, n_table_rows, err);
    else if (dtype == THN_F32)
        thn_launch(token_gate_kernel<float>, blocks, 256, 0, stream, (float*)out, (const float*)z, (const float*)table, tokens,
                   rows, dim, (long long)table_width, column0, n_table_rows, err);
    else
        THN_CHECK_ARG(false, "token_gate: unknown dtype %d", dtype);
    return thn_launch_status("token_gate");
}

// x [rows, width] and w [dim, width] bfloat16, 16-byte aligned, width a multiple of eight.  With h (float32
// [rows, width]) instead of x: the row is h + scale1 first + scale2 second (second and scale2 may be null).
THN_API int thn_token_gate_product_bf16(void* out, const void* x, const float* h, const void* first, const float* scale1,
                                        const void* second, const float* scale2, const void* w, const void* table,
                                        const int* tokens, int rows, int width, int dim, int table_width, int column0,
                                        int n_table_rows, int* err, cudaStream_t stream) {
    THN_CHECK_ARG(rows >= 0 && dim > 0 && width > 0 && width % 8 == 0 && column0 >= 0 && column0 + dim <= table_width &&
                      n_table_rows > 0,
                  "token_gate_product: bad sizes rows=%d width=%d dim=%d", rows, width, dim);
    THN_CHECK_ARG((x == nullptr) != (h == nullptr), "token_gate_product: a row, or a stream with what is pending (rows=%d)", rows);
    THN_CHECK_ARG(h == nullptr || (first && scale1 && (second == nullptr) == (scale2 == nullptr)),
                  "token_gate_product: pending outputs come with their factors (rows=%d)", rows);
    THN_CHECK_ARG((((uintptr_t)x | (uintptr_t)w | (uintptr_t)h | (uintptr_t)first | (uintptr_t)scale1 | (uintptr_t)second |
                    (uintptr_t)scale2) & 15) == 0, "token_gate_product: operands must be 16-byte aligned (rows=%d)", rows);
    if (rows == 0) return THN_OK;
    const int groups = (dim + 3) / 4, want = (2 * 148 + rows - 1) / rows;
    const dim3 grid(rows, groups < want ? groups : want);
    const Pending pending{h, (const __nv_bfloat16*)first, (const __nv_bfloat16*)second, scale1, scale2};
    const size_t smem = h ? (size_t)width * 2 : 0;
    THN_UNSUPPORTED_IF(smem > 40 * 1024, "token_gate_product: rows of %d values do not fit shared memory", width);
    if (h)
        thn_launch(token_gate_product_kernel<true>, grid, kProductThreads, smem, stream, (__nv_bfloat16*)out,
                   (const __nv_bfloat16*)x, pending, (const __nv_bfloat16*)w, (const __nv_bfloat16*)table, tokens, dim, width / 8,
                   (long long)table_width, column0, n_table_rows, err);
    else
        thn_launch(token_gate_product_kernel<false>, grid, kProductThreads, smem, stream, (__nv_bfloat16*)out,
                   (const __nv_bfloat16*)x, pending, (const __nv_bfloat16*)w, (const __nv_bfloat16*)table, tokens, dim, width / 8,
                   (long long)table_width, column0, n_table_rows, err);
    return thn_launch_status("token_gate_product");
}
