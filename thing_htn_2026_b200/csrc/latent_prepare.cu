// Preparation of attention whose keys and values are read out of one low-rank latent per token.
//
// A token's projected row holds, among others, a latent part of `rank` entries and one shared
// key part of `rot` entries that is to be rotated by the token's position.
//
//   latent_norm      c = latent / sqrt(mean(latent^2) + eps) * w   -> [rows, rank], the operand of
//                    the up-projection that gives every head's unrotated key and its value.  Where
//                    the queries are read out of a latent of their own, both are normalised in one launch.
//   latent_assemble  from the row's queries [heads][plain | rot], the up-projection's result
//                    [heads * plain keys | heads * values] and the shared key part: queries with
//                    their last `rot` entries rotated; per head the key [plain | rotated shared
//                    part] and the value, written to the paged cache (keys of plain + rot
//                    entries, values of a size of their own).
//
// The rotation pairs entry 2i with entry 2i + 1 of the rotated part (interleaved) or entry i with
// entry i + rot / 2 (half): (a, b) with angle t becomes (a cos t - b sin t, b cos t + a sin t); cos and sin come from tables [positions, rot / 2]
// (which may carry a common magnitude).  float32 between the load and the one rounding at the
// store; what is only copied is copied as it is.  One block per row.
#include "common.cuh"

namespace {

// One latent of a projected row: where it starts in the row, its size, its gain and its output.
struct Latent {
    void* out;
    const float* gain;
    long long offset;
    int rank;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_norm_kernel(Latent one, Latent two, const T* __restrict__ src,
                                                          long long src_stride, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[33];
    const Latent l = blockIdx.y ? two : one;
    const T* row = src + (size_t)blockIdx.x * src_stride + l.offset;
    T* out = (T*)l.out + (size_t)blockIdx.x * l.rank;
    float ss = 0.f;
    for (int i = threadIdx.x; i < l.rank; i += blockDim.x) {
        const float v = to_f32<T>(row[i]);
        ss += v * v;
    }
    const float r = 1.0f / sqrtf(block_sum(ss, scratch) / (float)l.rank + eps);
    for (int i = threadIdx.x; i < l.rank; i += blockDim.x) out[i] = from_f32<T>(to_f32<T>(row[i]) * r * l.gain[i]);
}

// The same for bfloat16 in 16-byte pieces; a thread's first piece stays in registers between the two passes.
__global__ void __launch_bounds__(128) latent_norm_vec_kernel(Latent one, Latent two, const __nv_bfloat16* __restrict__ src,
                                                              long long src_stride, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[33];
    const Latent l = blockIdx.y ? two : one;
    const uint4* row = reinterpret_cast<const uint4*>(src + (size_t)blockIdx.x * src_stride + l.offset);
    uint4* out = reinterpret_cast<uint4*>((__nv_bfloat16*)l.out + (size_t)blockIdx.x * l.rank);
    const int pieces = l.rank / 8;
    uint4 first = make_uint4(0, 0, 0, 0);
    float ss = 0.f;
    for (int i = threadIdx.x; i < pieces; i += 128) {
        const uint4 raw = row[i];
        if (i < 128) first = raw;
        const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 v = __bfloat1622float2(x[j]);
            ss += v.x * v.x + v.y * v.y;
        }
    }
    const float r = 1.0f / sqrtf(block_sum(ss, scratch) / (float)l.rank + eps);
    for (int i = threadIdx.x; i < pieces; i += 128) {
        const uint4 raw = i < 128 ? first : row[i];
        const float4 g0 = reinterpret_cast<const float4*>(l.gain)[2 * i], g1 = reinterpret_cast<const float4*>(l.gain)[2 * i + 1];
        const float g[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
        const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&raw);
        uint4 packed;
        __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 v = __bfloat1622float2(x[j]);
            o[j] = __floats2bfloat162_rn(v.x * r * g[2 * j], v.y * r * g[2 * j + 1]);
        }
        out[i] = packed;
    }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_assemble_kernel(
    T* __restrict__ q_out, const T* __restrict__ q_src, long long q_stride, const T* __restrict__ shared_src,
    long long shared_stride, const T* __restrict__ up, const float* __restrict__ cos_tab,
    const float* __restrict__ sin_tab, int table_len, const int* __restrict__ row_slot, const int* __restrict__ row_pos,
    PagedKV kv, int n_heads, int plain, int rot, int interleaved, int value_src, int* __restrict__ err) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x;
    const int pos = row_pos[m];
    const int D = plain + rot, DV = kv.value_dim > 0 ? kv.value_dim : kv.head_dim, half = rot / 2;
    if (pos >= table_len) {
        if (threadIdx.x == 0 && err) atomicOr(err, THN_ERR_POSITION_RANGE);
        return;
    }
    const int page = kv.block_table[(size_t)row_slot[m] * kv.bt_stride + pos / kv.page_size];
    const int in_page = pos % kv.page_size;
    if (page < 0 && threadIdx.x == 0 && err) atomicOr(err, THN_ERR_PAGE_UNMAPPED);
    const float* c_row = cos_tab + (size_t)pos * half;
    const float* s_row = sin_tab + (size_t)pos * half;
    const T* q_row = q_src + (size_t)m * q_stride;
    const T* k_shared = shared_src + (size_t)m * shared_stride;
    const T* up_row = up + (size_t)m * n_heads * (plain + value_src);
    T* cache = (T*)kv.base;
    // pair i of a rotated part: its first entry, and how far behind it the second one lies
    const int first = interleaved ? 2 : 1, apart = interleaved ? 1 : half;

    // queries: the plain part as it is, the rest rotated
    for (int e = threadIdx.x; e < n_heads * plain; e += blockDim.x) {
        const int h = e / plain, d = e - h * plain;
        q_out[((size_t)m * n_heads + h) * D + d] = q_row[h * D + d];
    }
    for (int e = threadIdx.x; e < n_heads * half; e += blockDim.x) {
        const int h = e / half, i = e - h * half;
        const T* src = q_row + h * D + plain + first * i;
        const float a = to_f32<T>(src[0]), b = to_f32<T>(src[apart]);
        const float c = c_row[i], s = s_row[i];
        T* dst = q_out + ((size_t)m * n_heads + h) * D + plain + first * i;
        dst[0] = from_f32<T>(a * c - b * s);
        dst[apart] = from_f32<T>(b * c + a * s);
    }
    if (page < 0) return;
    // keys: every head's plain part from the up-projection, then the shared part, rotated
    for (int e = threadIdx.x; e < n_heads * plain; e += blockDim.x) {
        const int h = e / plain, d = e - h * plain;
        cache[kv_offset_sized(kv, page, 0, h, in_page) + d] = up_row[e];
    }
    for (int e = threadIdx.x; e < n_heads * half; e += blockDim.x) {
        const int h = e / half, i = e - h * half;
        const float a = to_f32<T>(k_shared[first * i]), b = to_f32<T>(k_shared[first * i + apart]);
        const float c = c_row[i], s = s_row[i];
        T* dst = cache + kv_offset_sized(kv, page, 0, h, in_page) + plain + first * i;
        dst[0] = from_f32<T>(a * c - b * s);
        dst[apart] = from_f32<T>(b * c + a * s);
    }
    // values: the cache's rows may be wider than the values (padded to the keys' size); the rest is zero
    for (int e = threadIdx.x; e < n_heads * DV; e += blockDim.x) {
        const int h = e / DV, d = e - h * DV;
        cache[kv_offset_sized(kv, page, 1, h, in_page) + d] =
            d < value_src ? up_row[n_heads * plain + h * value_src + d] : from_f32<T>(0.f);
    }
}

// The same for bfloat16 where every part is whole 16-byte pieces (eight entries): a thread takes a piece,
// or, for half pairs, the two pieces that turn together.
__device__ __forceinline__ void turn_eight(const uint4& first, const uint4& second, const float* __restrict__ c,
                                           const float* __restrict__ s, uint4& out_first, uint4& out_second) {
    const __nv_bfloat162* a2 = reinterpret_cast<const __nv_bfloat162*>(&first);
    const __nv_bfloat162* b2 = reinterpret_cast<const __nv_bfloat162*>(&second);
    __nv_bfloat162* x2 = reinterpret_cast<__nv_bfloat162*>(&out_first);
    __nv_bfloat162* y2 = reinterpret_cast<__nv_bfloat162*>(&out_second);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float2 a = __bfloat1622float2(a2[j]), b = __bfloat1622float2(b2[j]);
        const float c0 = c[2 * j], c1 = c[2 * j + 1], s0 = s[2 * j], s1 = s[2 * j + 1];
        x2[j] = __floats2bfloat162_rn(a.x * c0 - b.x * s0, a.y * c1 - b.y * s1);
        y2[j] = __floats2bfloat162_rn(b.x * c0 + a.x * s0, b.y * c1 + a.y * s1);
    }
}
__device__ __forceinline__ uint4 turn_four_pairs(const uint4& in, const float* __restrict__ c, const float* __restrict__ s) {
    const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&in);
    uint4 out;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float2 v = __bfloat1622float2(p2[j]);
        o2[j] = __floats2bfloat162_rn(v.x * c[j] - v.y * s[j], v.y * c[j] + v.x * s[j]);
    }
    return out;
}

__global__ void __launch_bounds__(256) latent_assemble_vec_kernel(
    __nv_bfloat16* __restrict__ q_out, const __nv_bfloat16* __restrict__ q_src, long long q_stride,
    const __nv_bfloat16* __restrict__ shared_src, long long shared_stride, const __nv_bfloat16* __restrict__ up,
    const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, int table_len, const int* __restrict__ row_slot,
    const int* __restrict__ row_pos, PagedKV kv, int n_heads, int plain, int rot, int interleaved, int value_src,
    int* __restrict__ err) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x, pos = row_pos[m];
    const int D = plain + rot, DV = kv.value_dim > 0 ? kv.value_dim : kv.head_dim, half = rot / 2;
    if (pos >= table_len) {
        if (threadIdx.x == 0 && err) atomicOr(err, THN_ERR_POSITION_RANGE);
        return;
    }
    const int page = kv.block_table[(size_t)row_slot[m] * kv.bt_stride + pos / kv.page_size];
    const int in_page = pos % kv.page_size;
    if (page < 0 && threadIdx.x == 0 && err) atomicOr(err, THN_ERR_PAGE_UNMAPPED);
    const float* c_row = cos_tab + (size_t)pos * half;
    const float* s_row = sin_tab + (size_t)pos * half;
    const __nv_bfloat16* q_row = q_src + (size_t)m * q_stride;
    const __nv_bfloat16* k_shared = shared_src + (size_t)m * shared_stride;
    const __nv_bfloat16* up_row = up + (size_t)m * n_heads * (plain + value_src);
    auto piece = [](const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); };
    auto put = [](__nv_bfloat16* p, const uint4& v) { *reinterpret_cast<uint4*>(p) = v; };
    __nv_bfloat16* cache = page < 0 ? nullptr : (__nv_bfloat16*)kv.base;
    const long long keys0 = page < 0 ? 0 : kv_offset_sized(kv, page, 0, 0, in_page);
    const long long values0 = page < 0 ? 0 : kv_offset_sized(kv, page, 1, 0, in_page);
    const long long key_step = (long long)kv.page_size * D, value_step = (long long)kv.page_size * DV;
    // work items of a head: plain pieces, turned pieces (pairs of them for half pairs), value pieces
    const int plain_items = plain / 8, turned_items = interleaved ? rot / 8 : half / 8, value_items = DV / 8;
    const int per_head = plain_items + turned_items + value_items;
    for (int item = blockIdx.y * blockDim.x + threadIdx.x; item < n_heads * per_head; item += gridDim.y * blockDim.x) {
        const int h = item / per_head, i = item - h * per_head;
        const __nv_bfloat16* q = q_row + (size_t)h * D;
        __nv_bfloat16* dst = q_out + ((size_t)m * n_heads + h) * D;
        __nv_bfloat16* key = cache ? cache + keys0 + h * key_step : nullptr;
        if (i < plain_items) {
            put(dst + i * 8, piece(q + i * 8));
            if (key) put(key + i * 8, piece(up_row + (size_t)h * plain + i * 8));
        } else if (i < plain_items + turned_items) {
            const int j = (i - plain_items) * 8;
            if (interleaved) {
                put(dst + plain + j, turn_four_pairs(piece(q + plain + j), c_row + j / 2, s_row + j / 2));
                if (key) put(key + plain + j, turn_four_pairs(piece(k_shared + j), c_row + j / 2, s_row + j / 2));
            } else {
                uint4 x, y;
                turn_eight(piece(q + plain + j), piece(q + plain + half + j), c_row + j, s_row + j, x, y);
                put(dst + plain + j, x);
                put(dst + plain + half + j, y);
                if (key) {
                    turn_eight(piece(k_shared + j), piece(k_shared + half + j), c_row + j, s_row + j, x, y);
                    put(key + plain + j, x);
                    put(key + plain + half + j, y);
                }
            }
        } else if (cache) {
            const int j = (i - plain_items - turned_items) * 8;
            put(cache + values0 + h * value_step + j,
                j < value_src ? piece(up_row + (size_t)n_heads * plain + (size_t)h * value_src + j) : make_uint4(0, 0, 0, 0));
        }
    }
}

}  // namespace

// src: rows of the activation type, src_stride elements apart, with a latent of `rank` entries from column
// `offset` and, if out2 is given, another one of rank2 from offset2; gains float32 [rank]; out [rows, rank] of
// the activation type.
THN_API int thn_latent_norm(void* out, long long offset, const float* gain, int rank, void* out2, long long offset2,
                            const float* gain2, int rank2, const void* src, long long src_stride, float eps, int rows, int dtype,
                            cudaStream_t stream) {
    THN_CHECK_ARG(rows >= 0 && rank > 0 && offset >= 0 && src_stride >= offset + rank && eps > 0.f && gain, "latent_norm: bad arguments");
    THN_CHECK_ARG(out2 == nullptr || (rank2 > 0 && offset2 >= 0 && src_stride >= offset2 + rank2 && gain2),
                  "latent_norm: bad arguments of the second latent");
    if (rows == 0) return THN_OK;
    const Latent one{out, gain, offset, rank}, two{out2, gain2, offset2, rank2};
    const dim3 grid(rows, out2 ? 2 : 1);
    const bool whole = ((rank | (out2 ? rank2 : 0) | (int)(src_stride % 8) | (int)(offset % 8) | (int)(out2 ? offset2 % 8 : 0)) % 8) == 0 &&
                       (((uintptr_t)out | (uintptr_t)out2 | (uintptr_t)src | (uintptr_t)gain | (uintptr_t)gain2) & 15) == 0;
    if (dtype == THN_BF16 && whole)
        thn_launch(latent_norm_vec_kernel, grid, 128, 0, stream, one, two, (const __nv_bfloat16*)src, src_stride, eps);
    else if (dtype == THN_F32)
        thn_launch(latent_norm_kernel<float>, grid, 128, 0, stream, one, two, (const float*)src, src_stride, eps);
    else if (dtype == THN_BF16)
        thn_launch(latent_norm_kernel<__nv_bfloat16>, grid, 128, 0, stream, one, two, (const __nv_bfloat16*)src, src_stride, eps);
    else
        THN_CHECK_ARG(false, "latent_norm: unknown dtype %d", dtype);
    return thn_launch_status("latent_norm");
}

// q_src: [heads][plain + rot] per row, rows q_stride elements apart; shared_src: `rot` entries per
// row, rows shared_stride apart; up [rows, heads * plain + heads * value_src]; q_out
// [rows, heads * (plain + rot)].  The cache entry has `heads` kv heads, keys of plain + rot and
// values of value_dim >= value_src entries (what lies beyond a value is written as zero).
THN_API int thn_latent_assemble(void* q_out, const void* q_src, long long q_stride, const void* shared_src,
                                long long shared_stride, const void* up, const float* cos_tab, const float* sin_tab,
                                int table_len, const int* row_slot, const int* row_pos, void* kv_base,
                                const int* block_table, int bt_stride, int page_size, int n_rows, int n_heads, int plain,
                                int rot, int interleaved, int value_dim, int value_src, int dtype, int* err,
                                cudaStream_t stream) {
    THN_CHECK_ARG(n_rows >= 0 && n_heads > 0 && plain >= 0 && rot >= 0 && rot % 2 == 0 && plain + rot > 0 && value_src > 0 &&
                      value_dim >= value_src && page_size > 0,
                  "latent_assemble: bad sizes");
    THN_CHECK_ARG(rot == 0 || (cos_tab && sin_tab), "latent_assemble: a rotated part needs tables");
    if (n_rows == 0) return THN_OK;
    const int D = plain + rot;
    PagedKV kv{kv_base, block_table, bt_stride, n_heads, page_size, D, value_dim == D ? 0 : value_dim};
    if (rot == 0) table_len = 1 << 30;
    const int turned = interleaved ? rot : rot / 2;
    if (dtype == THN_BF16 && plain % 8 == 0 && turned % 8 == 0 && value_dim % 8 == 0 && value_src % 8 == 0 && q_stride % 8 == 0 &&
        shared_stride % 8 == 0 &&
        (((uintptr_t)q_out | (uintptr_t)q_src | (uintptr_t)shared_src | (uintptr_t)up | (uintptr_t)kv_base) & 15) == 0) {
        const int items = n_heads * (plain / 8 + turned / 8 + value_dim / 8);
        const int per_row = n_rows >= 296 ? 1 : (items + 255) / 256;      // few rows: several blocks for each
        thn_launch(latent_assemble_vec_kernel, dim3(n_rows, per_row), 256, 0, stream, (__nv_bfloat16*)q_out,
                   (const __nv_bfloat16*)q_src, q_stride, (const __nv_bfloat16*)shared_src, shared_stride, (const __nv_bfloat16*)up,
                   cos_tab, sin_tab, table_len, row_slot, row_pos, kv, n_heads, plain, rot, interleaved, value_src, err);
        return thn_launch_status("latent_assemble");
    }
    if (dtype == THN_F32)
        thn_launch(latent_assemble_kernel<float>, n_rows, 256, 0, stream, (float*)q_out, (const float*)q_src, q_stride,
                   (const float*)shared_src, shared_stride, (const float*)up, cos_tab, sin_tab, table_len, row_slot, row_pos,
                   kv, n_heads, plain, rot, interleaved, value_src, err);
    else if (dtype == THN_BF16)
        thn_launch(latent_assemble_kernel<__nv_bfloat16>, n_rows, 256, 0, stream, (__nv_bfloat16*)q_out,
                   (const __nv_bfloat16*)q_src, q_stride, (const __nv_bfloat16*)shared_src, shared_stride,
                   (const __nv_bfloat16*)up, cos_tab, sin_tab, table_len, row_slot, row_pos, kv, n_heads, plain, rot, interleaved, value_src, err);
    else
        THN_CHECK_ARG(false, "latent_assemble: unknown dtype %d", dtype);
    return thn_launch_status("latent_assemble");
}
