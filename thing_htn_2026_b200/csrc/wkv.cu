// Time mixing (RWKV): a recurrent token mixer whose projections read blends of a token and the one
// before it.  Per head a matrix S [dim, dim], zero at a sequence's start, and for every token with
// receptance r, key k, value v, decay w in (0, 1) per key channel and a bonus u per key channel
//
//     o = (S + diag(u) k v^T)^T r          S <- diag(w) S + k v^T          w = exp(-exp(z + w0))
//
//   token_shift      the blends: out[s] = h + (h' - h) mu[s] for each of the projections s, h' the row
//                    of the token before: the row above in the packed step or, for the first row
//                    that a sequence brings, what the sequence's last step left in `shift` (zeros at
//                    the start).  The block of a sequence's first row also leaves its last row there:
//                    a column is read and then written by one thread.
//   tanh_rows        the activation between the two products of the decay.
//   wkv_prepare      float32 rows for the shared recurrence (linear_attention.cuh, kBonusRead): k, r and
//                    w per key channel, v, and the token's own share b = sum_d r_d u_d k_d.  One warp
//                    per (row, head).
//   wkv_decode       a single token per sequence, from the products to the operand of the output
//                    projection in one kernel: the second product of the decay (it has few channels)
//                    with the tanh ahead of it, the recurrence, the norm of each head's read-out, its
//                    gain and the silu gate.  One block per (row, head).
//
// float32 after the loads: the blends, the decay with both exponentials, the state, the sums, the
// norm.  With float32 activations the exponentials are computed in double and rounded once.
#include <math.h>

#include "linear_attention.cuh"

namespace {

// exp(-exp(x)): a decay from its unbounded input
template <typename T> __device__ __forceinline__ float double_exp(float x) { return expf(-expf(x)); }
template <> __device__ __forceinline__ float double_exp<float>(float x) { return (float)exp(-exp((double)x)); }
template <typename T> __device__ __forceinline__ float tanh_of(float x) { return tanhf(x); }
template <> __device__ __forceinline__ float tanh_of<float>(float x) { return (float)tanh((double)x); }

// The sequence of packed row m: the last i with cu_seqlens[i] <= m.
__device__ __forceinline__ int sequence_of_row(const int* __restrict__ cu_seqlens, int n_seqs, int m) {
    int lo = 0, hi = n_seqs - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (cu_seqlens[mid] <= m) lo = mid; else hi = mid - 1;
    }
    return lo;
}

template <typename T>
__global__ void __launch_bounds__(256) token_shift_kernel(T* __restrict__ out, const T* __restrict__ x,
                                                          const float* __restrict__ mu, T* __restrict__ shift,
                                                          const int* __restrict__ row_slot, const int* __restrict__ row_pos,
                                                          const int* __restrict__ cu_seqlens, const int* __restrict__ seq_lens,
                                                          int n_rows, int n_seqs, int width, int n_mix) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x;
    const int slot = row_slot[m], pos = row_pos[m];
    const bool first = pos == seq_lens[slot];            // the first row its sequence brings
    const T* own = x + (size_t)m * width;
    T* kept = shift + (size_t)slot * width;
    const T* last = nullptr;
    if (first) last = x + (size_t)(cu_seqlens[sequence_of_row(cu_seqlens, n_seqs, m) + 1] - 1) * width;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < width; c += gridDim.y * blockDim.x) {
        const float h = to_f32<T>(own[c]);
        float before;
        if (first) {
            before = pos == 0 ? 0.f : to_f32<T>(kept[c]);
            kept[c] = last[c];
        } else {
            before = to_f32<T>(own[c - width]);
        }
        for (int s = 0; s < n_mix; ++s)
            out[((size_t)s * n_rows + m) * width + c] = from_f32<T>(h + (before - h) * mu[(size_t)s * width + c]);
    }
}

// The same, eight bfloat16 columns per thread (16-byte accesses).
__global__ void __launch_bounds__(128) token_shift_bf16_vec_kernel(
    __nv_bfloat16* __restrict__ out, const __nv_bfloat16* __restrict__ x, const float* __restrict__ mu,
    __nv_bfloat16* __restrict__ shift, const int* __restrict__ row_slot, const int* __restrict__ row_pos,
    const int* __restrict__ cu_seqlens, const int* __restrict__ seq_lens, int n_rows, int n_seqs, int width, int n_mix) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
    if (c >= width) return;
    const int slot = row_slot[m], pos = row_pos[m];
    const __nv_bfloat16* own = x + (size_t)m * width + c;
    const uint4 raw = *reinterpret_cast<const uint4*>(own);
    uint4 raw_before = make_uint4(0, 0, 0, 0);
    if (pos == seq_lens[slot]) {
        __nv_bfloat16* kept = shift + (size_t)slot * width + c;
        if (pos != 0) raw_before = *reinterpret_cast<const uint4*>(kept);
        const int last = cu_seqlens[sequence_of_row(cu_seqlens, n_seqs, m) + 1] - 1;
        *reinterpret_cast<uint4*>(kept) = *reinterpret_cast<const uint4*>(x + (size_t)last * width + c);
    } else {
        raw_before = *reinterpret_cast<const uint4*>(own - width);
    }
    float h[8], step[8];
    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
    const __nv_bfloat162* b2 = reinterpret_cast<const __nv_bfloat162*>(&raw_before);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 a = __bfloat1622float2(h2[i]), b = __bfloat1622float2(b2[i]);
        h[2 * i] = a.x; h[2 * i + 1] = a.y;
        step[2 * i] = b.x - a.x; step[2 * i + 1] = b.y - a.y;
    }
    for (int s = 0; s < n_mix; ++s) {
        const float4 m0 = *reinterpret_cast<const float4*>(mu + (size_t)s * width + c);
        const float4 m1 = *reinterpret_cast<const float4*>(mu + (size_t)s * width + c + 4);
        uint4 packed;
        __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&packed);
        o2[0] = __floats2bfloat162_rn(h[0] + step[0] * m0.x, h[1] + step[1] * m0.y);
        o2[1] = __floats2bfloat162_rn(h[2] + step[2] * m0.z, h[3] + step[3] * m0.w);
        o2[2] = __floats2bfloat162_rn(h[4] + step[4] * m1.x, h[5] + step[5] * m1.y);
        o2[3] = __floats2bfloat162_rn(h[6] + step[6] * m1.z, h[7] + step[7] * m1.w);
        *reinterpret_cast<uint4*>(out + ((size_t)s * n_rows + m) * width + c) = packed;
    }
}

template <typename T>
__global__ void tanh_rows_kernel(T* __restrict__ out, const float* __restrict__ x, long long n) {
    pdl_launch_dependents();
    pdl_wait();
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (e < n) out[e] = from_f32<T>(tanh_of<T>(x[e]));
}

constexpr int kPrepareWarps = 4;

// prepared [rows][heads][k: kp | r: kp | w: kp | v: vp | b, 0, 0, 0], padded with zeros.
template <typename T>
__global__ void __launch_bounds__(kPrepareWarps * 32) wkv_prepare_kernel(
    float* __restrict__ prepared, const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v,
    const float* __restrict__ z, const float* __restrict__ w0, const float* __restrict__ u, long long n_units, int n_heads,
    int dim, int kp, int vp) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * kPrepareWarps + (threadIdx.x >> 5);
    if (unit >= n_units) return;
    const int head = (int)(unit % n_heads);
    const size_t at = (size_t)unit * dim;                       // (row * heads + head) * dim
    float* dst = prepared + (size_t)unit * (3 * kp + vp + kRecurrenceTail);
    float share = 0.f;
    for (int d = lane; d < kp; d += 32) {
        const bool in = d < dim;
        const float kd = in ? to_f32<T>(k[at + d]) : 0.f, rd = in ? to_f32<T>(r[at + d]) : 0.f;
        dst[d] = kd;
        dst[kp + d] = rd;
        dst[2 * kp + d] = in ? double_exp<T>(z[at + d] + w0[head * dim + d]) : 0.f;
        if (in) share += rd * u[head * dim + d] * kd;
    }
    for (int d = lane; d < vp; d += 32) dst[3 * kp + d] = d < dim ? to_f32<T>(v[at + d]) : 0.f;
    share = warp_sum(share);
    if (lane < kRecurrenceTail) dst[3 * kp + vp + lane] = lane == 0 ? share : 0.f;
}

constexpr int kDecodeThreads = 256;
constexpr int kDecodeLanes = 8;            // lanes that share a column of S

// Shared memory: r, k, v, w [dim] each, tanh'd low-rank input [rank], the read-out [dim].
template <typename T>
__global__ void __launch_bounds__(kDecodeThreads) wkv_decode_kernel(
    T* __restrict__ out, float* __restrict__ state, const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v,
    const T* __restrict__ gate, const float* __restrict__ low, int rank, const T* __restrict__ w2, const float* __restrict__ w0,
    const float* __restrict__ u, const float* __restrict__ gain, float eps, const int* __restrict__ row_slot, int n_heads,
    int dim) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float mem[];
    __shared__ float scratch[33];
    float *rs = mem, *ks = mem + dim, *vs = mem + 2 * dim, *ws = mem + 3 * dim, *os = mem + 4 * dim, *ls = mem + 5 * dim;
    const int head = blockIdx.x, row = blockIdx.y;
    const size_t at = ((size_t)row * n_heads + head) * dim;
    float share = 0.f;
    for (int d = threadIdx.x; d < dim; d += kDecodeThreads) {
        rs[d] = to_f32<T>(r[at + d]);
        ks[d] = to_f32<T>(k[at + d]);
        vs[d] = to_f32<T>(v[at + d]);
        share += rs[d] * u[head * dim + d] * ks[d];
    }
    for (int i = threadIdx.x; i < rank; i += kDecodeThreads) ls[i] = rnd<T>(tanh_of<T>(low[(size_t)row * rank + i]));
    share = block_sum(share, scratch);                 // (its barriers also order the stores above)
    {
        // the decay's second product: four threads per key channel
        const int part = threadIdx.x & 3;
        for (int d0 = 0; d0 < dim; d0 += kDecodeThreads / 4) {
            const int d = d0 + (threadIdx.x >> 2);
            float z = 0.f;
            if (d < dim) {
                const T* wr = w2 + ((size_t)head * dim + d) * rank;
                for (int i = part; i < rank; i += 4) z += to_f32<T>(wr[i]) * ls[i];
            }
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            z += __shfl_xor_sync(0xffffffffu, z, 2);
            if (part == 0 && d < dim) ws[d] = double_exp<T>(z + w0[head * dim + d]);
        }
    }
    __syncthreads();
    float* S = state + ((size_t)row_slot[row] * n_heads + head) * dim * dim;
    const int lane = threadIdx.x % kDecodeLanes, group = threadIdx.x / kDecodeLanes;
    constexpr int kGroups = kDecodeThreads / kDecodeLanes;
    const bool vec = dim % 4 == 0;
    for (int e0 = 0; e0 < dim; e0 += kGroups) {
        const int e = e0 + group;
        float part = 0.f;
        if (e < dim) {
            float* col = S + (size_t)e * dim;
            const float ve = vs[e];
            if (vec) {
                for (int d = lane * 4; d < dim; d += kDecodeLanes * 4) {
                    float4 s = *reinterpret_cast<const float4*>(col + d);
                    const float4 rd = *reinterpret_cast<const float4*>(rs + d), kd = *reinterpret_cast<const float4*>(ks + d);
                    const float4 wd = *reinterpret_cast<const float4*>(ws + d);
                    part += s.x * rd.x + s.y * rd.y + s.z * rd.z + s.w * rd.w;
                    s.x = wd.x * s.x + kd.x * ve;
                    s.y = wd.y * s.y + kd.y * ve;
                    s.z = wd.z * s.z + kd.z * ve;
                    s.w = wd.w * s.w + kd.w * ve;
                    *reinterpret_cast<float4*>(col + d) = s;
                }
            } else {
                for (int d = lane; d < dim; d += kDecodeLanes) {
                    const float s = col[d];
                    part += s * rs[d];
                    col[d] = ws[d] * s + ks[d] * ve;
                }
            }
        }
#pragma unroll
        for (int off = kDecodeLanes / 2; off > 0; off >>= 1) part += __shfl_xor_sync(0xffffffffu, part, off);
        if (lane == 0 && e < dim) os[e] = part + share * vs[e];
    }
    __syncthreads();
    float ss = 0.f;
    for (int e = threadIdx.x; e < dim; e += kDecodeThreads) ss += os[e] * os[e];
    const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)dim + eps);
    for (int e = threadIdx.x; e < dim; e += kDecodeThreads)
        out[at + e] = from_f32<T>(os[e] * rstd * gain[head * dim + e] * silu_of<T>(to_f32<T>(gate[at + e])));
}

}  // namespace

// x [rows, width]; mu float32 [n_mix, width]; out [n_mix, rows, width]; shift [slots, width] of the
// activation type, read and updated; seq_lens int32 [slots]: the tokens each slot held before the
// step; the rows of sequence i of the step are [cu_seqlens[i], cu_seqlens[i + 1]).
THN_API int thn_token_shift(void* out, const void* x, const float* mu, void* shift, const int* row_slot, const int* row_pos,
                            const int* cu_seqlens, const int* seq_lens, int n_rows, int n_seqs, int width, int n_mix, int dtype,
                            cudaStream_t stream) {
    THN_CHECK_ARG(n_rows >= 0 && n_seqs >= 0 && width > 0 && n_mix > 0, "token_shift: bad sizes");
    if (n_rows == 0) return THN_OK;
    if (dtype == THN_BF16 && width % 8 == 0 && (((uintptr_t)out | (uintptr_t)x | (uintptr_t)mu | (uintptr_t)shift) & 15) == 0) {
        thn_launch(token_shift_bf16_vec_kernel, dim3(n_rows, (width / 8 + 127) / 128), 128, 0, stream, (__nv_bfloat16*)out,
                   (const __nv_bfloat16*)x, mu, (__nv_bfloat16*)shift, row_slot, row_pos, cu_seqlens, seq_lens, n_rows, n_seqs,
                   width, n_mix);
        return thn_launch_status("token_shift");
    }
    const dim3 grid(n_rows, (width + 1023) / 1024);
    if (dtype == THN_F32)
        thn_launch(token_shift_kernel<float>, grid, 256, 0, stream, (float*)out, (const float*)x, mu, (float*)shift, row_slot,
                   row_pos, cu_seqlens, seq_lens, n_rows, n_seqs, width, n_mix);
    else if (dtype == THN_BF16)
        thn_launch(token_shift_kernel<__nv_bfloat16>, grid, 256, 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)x, mu,
                   (__nv_bfloat16*)shift, row_slot, row_pos, cu_seqlens, seq_lens, n_rows, n_seqs, width, n_mix);
    else
        THN_CHECK_ARG(false, "token_shift: unknown dtype %d", dtype);
    return thn_launch_status("token_shift");
}

// out (activation type) = tanh(x), n entries.
THN_API int thn_tanh_rows(void* out, const float* x, long long n, int dtype, cudaStream_t stream) {
    THN_CHECK_ARG(n >= 0, "tanh_rows: bad size");
    if (n == 0) return THN_OK;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (dtype == THN_F32) thn_launch(tanh_rows_kernel<float>, blocks, 256, 0, stream, (float*)out, x, n);
    else if (dtype == THN_BF16) thn_launch(tanh_rows_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (__nv_bfloat16*)out, x, n);
    else THN_CHECK_ARG(false, "tanh_rows: unknown dtype %d", dtype);
    return thn_launch_status("tanh_rows");
}

// Floats of the scratch that thn_wkv needs for a step of n_rows rows.
THN_API long long thn_wkv_scratch_floats(int n_rows, int n_heads, int dim) {
    return (long long)n_rows * n_heads * (3 * padded_keys(dim) + padded_values(dim) + kRecurrenceTail);
}

// o float32 [rows, heads, dim]; state float32 [slots, heads, dim (value), dim (key)], read and updated;
// r, k, v [rows, heads * dim] of the activation type; z float32 [rows, heads * dim] (the decay's input
// without its bias w0 float32 [heads * dim]); u float32 [heads, dim]; scratch float32, 16-byte aligned.
THN_API int thn_wkv(float* o, float* state, float* scratch, const void* r, const void* k, const void* v, const float* z,
                    const float* w0, const float* u, const int* cu_seqlens, const int* slots, int n_rows, int n_seqs,
                    int n_heads, int dim, int dtype, cudaStream_t stream) {
    THN_CHECK_ARG(n_rows >= 0 && n_seqs >= 0 && n_heads > 0 && dim > 0, "wkv: bad sizes");
    THN_UNSUPPORTED_IF(dim > 512, "wkv: heads of %d, at most 512", dim);
    THN_CHECK_ARG(scratch != nullptr && ((uintptr_t)scratch & 15) == 0, "wkv: scratch missing or unaligned");
    if (n_rows == 0 || n_seqs == 0) return THN_OK;
    const int kp = padded_keys(dim), vp = padded_values(dim), per = 3 * kp + vp + kRecurrenceTail;
    const long long units = (long long)n_rows * n_heads;
    const unsigned blocks = (unsigned)((units + kPrepareWarps - 1) / kPrepareWarps);
    if (dtype == THN_F32)
        thn_launch(wkv_prepare_kernel<float>, blocks, kPrepareWarps * 32, 0, stream, scratch, (const float*)r, (const float*)k,
                   (const float*)v, z, w0, u, units, n_heads, dim, kp, vp);
    else if (dtype == THN_BF16)
        thn_launch(wkv_prepare_kernel<__nv_bfloat16>, blocks, kPrepareWarps * 32, 0, stream, scratch, (const __nv_bfloat16*)r,
                   (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, z, w0, u, units, n_heads, dim, kp, vp);
    else
        THN_CHECK_ARG(false, "wkv: unknown dtype %d", dtype);
    return launch_recurrence(kBonusRead, RecurrenceArgs{o, state, scratch, per, n_heads, scratch + 3 * kp, per, nullptr, cu_seqlens,
                                                        slots, n_seqs, n_heads, dim, dim, 1.0f}, stream);
}

// One token per sequence.  r, k, v, gate, out [rows, heads * dim] of the activation type; low float32
// [rows, rank]: the decay's inner channels before the tanh; w2 [heads * dim, rank] of the activation
// type; gain float32 [heads * dim]; the rest as above.
THN_API int thn_wkv_decode(void* out, float* state, const void* r, const void* k, const void* v, const void* gate,
                           const float* low, int rank, const void* w2, const float* w0, const float* u, const float* gain,
                           float eps, const int* row_slot, int n_rows, int n_heads, int dim, int dtype, cudaStream_t stream) {
    THN_CHECK_ARG(n_rows >= 0 && n_heads > 0 && dim > 0 && rank > 0 && eps > 0.f, "wkv_decode: bad sizes");
    THN_UNSUPPORTED_IF(dim > 512 || rank > 4096 || n_rows > 65535, "wkv_decode: heads of %d, rank %d, %d rows", dim, rank, n_rows);
    if (n_rows == 0) return THN_OK;
    const size_t smem = (size_t)(5 * dim + rank) * sizeof(float);
    const dim3 grid(n_heads, n_rows);
    if (dtype == THN_F32)
        thn_launch(wkv_decode_kernel<float>, grid, kDecodeThreads, smem, stream, (float*)out, state, (const float*)r,
                   (const float*)k, (const float*)v, (const float*)gate, low, rank, (const float*)w2, w0, u, gain, eps, row_slot,
                   n_heads, dim);
    else if (dtype == THN_BF16)
        thn_launch(wkv_decode_kernel<__nv_bfloat16>, grid, kDecodeThreads, smem, stream, (__nv_bfloat16*)out, state,
                   (const __nv_bfloat16*)r, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, (const __nv_bfloat16*)gate, low,
                   rank, (const __nv_bfloat16*)w2, w0, u, gain, eps, row_slot, n_heads, dim);
    else
        THN_CHECK_ARG(false, "wkv_decode: unknown dtype %d", dtype);
    return thn_launch_status("wkv_decode");
}
