// State-space duality (Mamba-2): a recurrent token mixer.  Per head a matrix S [state, vdim], zero at a
// sequence's start, and for every token with an input x (vdim entries per head), B and C (state
// entries, shared by a group of neighbouring heads), one step size t and one decay a per head:
//
//     t = softplus(t_pre + bias_h)       a = exp(-rate_h t)
//     S <- a S + (t B) x^T               y = S^T C + D_h x
//
// x, B and C come out of one short causal convolution per channel with a bias and silu; the raw
// inputs of a sequence's last `taps` tokens stay in a ring [taps, channels], position p at p mod taps.
//
//   state_space_prepare   convolution, silu, step sizes and decays of a prompt's rows, into float32 rows
//                    for the shared recurrence (linear_attention.cuh, kSteppedDecay): [B | C] per row
//                    and group, [x | a, t] per row and head.  A thread takes four neighbouring
//                    channels over a run of rows, keeping the last raw inputs in registers.
//   state_space_decode    a single token per sequence: convolution, ring, step size, decay, recurrence
//                    and skip in one kernel, one block per (row, head).
//   gated_group_norm   y silu(z), divided by its root mean square over equal consecutive parts, times a
//                    gain: the gate comes before the norm.
//
// float32 after the loads; with float32 activations the exponentials and logarithms are computed in
// double and rounded once (exp_of, silu_of, softplus_of in common.cuh).
#include <math.h>

#include "linear_attention.cuh"

namespace {

constexpr int kRunRows = 8;          // rows per thread of the prepare kernel
constexpr int kPrepareThreads = 128;

struct SpaceShape {
    int n_heads, vdim, n_state, n_groups, taps;
    __host__ __device__ int inner() const { return n_heads * vdim; }
    __host__ __device__ int channels() const { return n_heads * vdim + 2 * n_groups * n_state; }
};

template <typename T> __device__ __forceinline__ float4 load_four(const T* p);
template <> __device__ __forceinline__ float4 load_four<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load_four<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ float4 load_up_to_four(const T* p, int n, bool vec) {
    if (vec) return load_four<T>(p);
    return make_float4(n > 0 ? to_f32<T>(p[0]) : 0.f, n > 1 ? to_f32<T>(p[1]) : 0.f, n > 2 ? to_f32<T>(p[2]) : 0.f,
                       n > 3 ? to_f32<T>(p[3]) : 0.f);
}
__device__ __forceinline__ void add_scaled(float4& acc, const float4& w, const float4& v) {
    acc.x += w.x * v.x; acc.y += w.y * v.y; acc.z += w.z * v.z; acc.w += w.w * v.w;
}

// keys [rows][groups][B: kp | C: kp], values [rows][heads][x: vp | a, t, 0, 0].  Work items of a row:
// heads * vp / 4 pieces of x, groups * 2 * kp / 4 pieces of B and C, one tail per head.
// TAPS 0: any number, every raw input loaded where it is used.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kPrepareThreads) state_space_prepare_kernel(
    float* __restrict__ keys, float* __restrict__ values, const T* __restrict__ proj, int proj_width, int offset,
    const float* __restrict__ conv_w, const float* __restrict__ conv_b, const T* __restrict__ ring,
    const float* __restrict__ dt_pre, const float* __restrict__ dt_bias, const float* __restrict__ rate,
    const int* __restrict__ row_slot, const int* __restrict__ row_pos, const int* __restrict__ seq_lens, int n_rows,
    SpaceShape shape, int kp, int vp, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    const int taps = TAPS > 0 ? TAPS : shape.taps;
    const int x_items = shape.n_heads * (vp / 4), bc_items = shape.n_groups * 2 * (kp / 4);
    const int item = blockIdx.x * kPrepareThreads + threadIdx.x;
    const int first_row = blockIdx.y * kRunRows, last_row = min(first_row + kRunRows, n_rows);
    const int value_stride = vp + kRecurrenceTail, channels = shape.channels();
    if (item >= x_items + bc_items + shape.n_heads) return;
    if (item >= x_items + bc_items) {                       // a head's step sizes and decays
        const int head = item - x_items - bc_items;
        const float bias = dt_bias[head], r = rate[head];
        for (int m = first_row; m < last_row; ++m) {
            const float t = softplus_of<T>(dt_pre[(size_t)m * shape.n_heads + head] + bias);
            *reinterpret_cast<float4*>(values + ((size_t)m * shape.n_heads + head) * value_stride + vp) =
                make_float4(exp_of<T>(-r * t), t, 0.f, 0.f);
        }
        return;
    }
    int channel, n;                                         // first source channel, how many of the four exist
    float* dst;
    size_t dst_stride;
    if (item < x_items) {
        const int head = item / (vp / 4), d = (item - head * (vp / 4)) * 4;
        channel = head * shape.vdim + d;
        n = shape.vdim - d;
        dst = values + (size_t)head * value_stride + d;
        dst_stride = (size_t)shape.n_heads * value_stride;
    } else {
        const int unit = (item - x_items) / (kp / 4), d = ((item - x_items) - unit * (kp / 4)) * 4;   // unit = group * 2 + which
        const int group = unit >> 1, which = unit & 1;
        channel = shape.inner() + (which * shape.n_groups + group) * shape.n_state + d;
        n = shape.n_state - d;
        dst = keys + (size_t)unit * kp + d;
        dst_stride = (size_t)shape.n_groups * 2 * kp;
    }
    dst += (size_t)first_row * dst_stride;
    if (n <= 0) {
        for (int m = first_row; m < last_row; ++m, dst += dst_stride) *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
        return;
    }
    const bool whole = vec && n >= 4;
    const float4 bias = load_up_to_four<float>(conv_b + channel, n, false);
    // a channel's taps are consecutive: four channels' weights for one tap are `taps` apart
    auto weight_of = [&](int j) {
        const float* w = conv_w + (size_t)channel * taps + j;
        return make_float4(w[0], n > 1 ? w[taps] : 0.f, n > 2 ? w[2 * taps] : 0.f, n > 3 ? w[3 * taps] : 0.f);
    };
    // the raw input `back` tokens before row m: from the step's rows, from the ring, or zero
    auto raw_of = [&](int m, int pos, int local, int slot, int back) {
        if (back > pos) return make_float4(0.f, 0.f, 0.f, 0.f);
        if (back <= local) return load_up_to_four<T>(proj + (size_t)(m - back) * proj_width + offset + channel, n, whole);
        return load_up_to_four<T>(ring + ((size_t)slot * taps + (pos - back) % taps) * channels + channel, n, whole);
    };
    constexpr int HELD = TAPS > 0 ? TAPS : 1;
    float4 w[HELD], past[HELD];                              // past[j]: the raw input TAPS - 1 - j tokens back
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < HELD; ++j) w[j] = weight_of(j);
    }
    for (int m = first_row; m < last_row; ++m, dst += dst_stride) {
        const int slot = row_slot[m], pos = row_pos[m];
        const int local = pos - seq_lens[slot];
        float4 acc = bias;
        if (TAPS > 0) {
            if (m == first_row || local == 0) {
#pragma unroll
                for (int j = 0; j < HELD - 1; ++j) past[j] = raw_of(m, pos, local, slot, HELD - 1 - j);
            } else {
#pragma unroll
                for (int j = 0; j < HELD - 1; ++j) past[j] = past[j + 1];
            }
            past[HELD - 1] = raw_of(m, pos, local, slot, 0);
#pragma unroll
            for (int j = 0; j < HELD; ++j) add_scaled(acc, w[j], past[j]);
        } else {
            for (int j = 0; j < taps; ++j) add_scaled(acc, weight_of(j), raw_of(m, pos, local, slot, taps - 1 - j));
        }
        *reinterpret_cast<float4*>(dst) = make_float4(silu_of<T>(acc.x), n > 1 ? silu_of<T>(acc.y) : 0.f,
                                                      n > 2 ? silu_of<T>(acc.z) : 0.f, n > 3 ? silu_of<T>(acc.w) : 0.f);
    }
}

constexpr int kDecodeThreads = 256;
constexpr int kDecodeLanes = 8;            // lanes that share a column of S

// Shared memory: B, C [n_state] each, x [vdim].
template <typename T>
__global__ void __launch_bounds__(kDecodeThreads) state_space_decode_kernel(
    float* __restrict__ y, float* __restrict__ state, const T* __restrict__ proj, int proj_width, int offset,
    const float* __restrict__ conv_w, const float* __restrict__ conv_b, T* __restrict__ ring, const float* __restrict__ dt_pre,
    const float* __restrict__ dt_bias, const float* __restrict__ rate, const float* __restrict__ skip,
    const int* __restrict__ row_slot, const int* __restrict__ row_pos, SpaceShape shape) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float mem[];
    const int N = shape.n_state, V = shape.vdim, taps = shape.taps, channels = shape.channels();
    const int padded = (N + 3) / 4 * 4;
    float *bs = mem, *cs = mem + padded, *xs = mem + 2 * padded;
    const int head = blockIdx.x, row = blockIdx.y;
    const int per_group = shape.n_heads / shape.n_groups, group = head / per_group;
    const int slot = row_slot[row], pos = row_pos[row];
    const T* src = proj + (size_t)row * proj_width + offset;
    T* slot_ring = ring + (size_t)slot * taps * channels;
    for (int i = threadIdx.x; i < V + 2 * N; i += kDecodeThreads) {
        const int c = i < V ? head * V + i
                            : shape.inner() + (i < V + N ? group * N + (i - V) : (shape.n_groups + group) * N + (i - V - N));
        const T raw = src[c];
        float acc = conv_b[c];
        for (int j = 0; j < taps - 1; ++j) {
            const int back = taps - 1 - j;
            if (back <= pos) acc += conv_w[(size_t)c * taps + j] * to_f32<T>(slot_ring[(size_t)((pos - back) % taps) * channels + c]);
        }
        acc += conv_w[(size_t)c * taps + taps - 1] * to_f32<T>(raw);
        // The entry that this token takes held the input of `taps` tokens ago, which no tap reads: blocks
        // that share B and C do not disturb one another.  The group's first head stores them.
        if (i < V || head == group * per_group) slot_ring[(size_t)(pos % taps) * channels + c] = raw;
        const float v = silu_of<T>(acc);
        if (i < V) xs[i] = v;
        else if (i < V + N) bs[i - V] = v;
        else cs[i - V - N] = v;
    }
    const float t = softplus_of<T>(dt_pre[(size_t)row * shape.n_heads + head] + dt_bias[head]);
    const float decay = exp_of<T>(-rate[head] * t), d_skip = skip[head];
    __syncthreads();
    float* S = state + ((size_t)slot * shape.n_heads + head) * V * N;
    const int lane = threadIdx.x % kDecodeLanes, column = threadIdx.x / kDecodeLanes;
    constexpr int kGroups = kDecodeThreads / kDecodeLanes;
    const bool vec = N % 4 == 0;
    for (int e0 = 0; e0 < V; e0 += kGroups) {
        const int e = e0 + column;
        float part = 0.f;
        if (e < V) {
            float* col = S + (size_t)e * N;
            const float tx = t * xs[e];
            if (vec) {
                for (int d = lane * 4; d < N; d += kDecodeLanes * 4) {
                    float4 s = *reinterpret_cast<const float4*>(col + d);
                    const float4 b = *reinterpret_cast<const float4*>(bs + d), c = *reinterpret_cast<const float4*>(cs + d);
                    s.x = decay * s.x + b.x * tx;
                    s.y = decay * s.y + b.y * tx;
                    s.z = decay * s.z + b.z * tx;
                    s.w = decay * s.w + b.w * tx;
                    part += s.x * c.x + s.y * c.y + s.z * c.z + s.w * c.w;
                    *reinterpret_cast<float4*>(col + d) = s;
                }
            } else {
                for (int d = lane; d < N; d += kDecodeLanes) {
                    const float s = decay * col[d] + bs[d] * tx;
                    part += s * cs[d];
                    col[d] = s;
                }
            }
        }
#pragma unroll
        for (int off = kDecodeLanes / 2; off > 0; off >>= 1) part += __shfl_xor_sync(0xffffffffu, part, off);
        if (lane == 0 && e < V) y[((size_t)row * shape.n_heads + head) * V + e] = part + d_skip * xs[e];
    }
}

// One block per (row, part), with as many threads as the part has pieces of four entries, up to 256.  The gated entries are computed twice, once for the sum of squares and
// once for the result; the second reading comes from the caches.
template <typename T>
__global__ void __launch_bounds__(256) gated_group_norm_kernel(T* __restrict__ out, const float* __restrict__ y,
                                                               const T* __restrict__ gate, long long gate_stride,
                                                               const float* __restrict__ gain, float eps, int width, int size,
                                                               int vec) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[33];
    const size_t base = (size_t)blockIdx.x * width + (size_t)blockIdx.y * size;
    const float* src = y + base;
    const T* g = gate + (size_t)blockIdx.x * gate_stride + (size_t)blockIdx.y * size;
    const float* w = gain + (size_t)blockIdx.y * size;
    T* dst = out + base;
    float ss = 0.f;
    if (vec) {
        constexpr int kKept = 4;                    // what fits stays in registers (parts up to sixteen entries a thread)
        float4 kept[kKept];
#pragma unroll
        for (int j = 0; j < kKept; ++j) {
            const int i = (j * (int)blockDim.x + (int)threadIdx.x) * 4;
            if (i < size) {
                const float4 v = *reinterpret_cast<const float4*>(src + i), z = load_four<T>(g + i);
                kept[j] = make_float4(v.x * silu_of<T>(z.x), v.y * silu_of<T>(z.y), v.z * silu_of<T>(z.z), v.w * silu_of<T>(z.w));
                ss += kept[j].x * kept[j].x + kept[j].y * kept[j].y + kept[j].z * kept[j].z + kept[j].w * kept[j].w;
            }
        }
        for (int i = (kKept * (int)blockDim.x + (int)threadIdx.x) * 4; i < size; i += (int)blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(src + i), z = load_four<T>(g + i);
            const float a = v.x * silu_of<T>(z.x), b = v.y * silu_of<T>(z.y), c = v.z * silu_of<T>(z.z), d = v.w * silu_of<T>(z.w);
            ss += a * a + b * b + c * c + d * d;
        }
        const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + eps);
        auto store = [&](int i, const float4& v) {
            const float4 gw = *reinterpret_cast<const float4*>(w + i);
            if constexpr (sizeof(T) == 2) {
                uint2 packed;
                *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(v.x * rstd * gw.x, v.y * rstd * gw.y);
                *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(v.z * rstd * gw.z, v.w * rstd * gw.w);
                *reinterpret_cast<uint2*>(dst + i) = packed;
            } else {
                *reinterpret_cast<float4*>(dst + i) = make_float4(v.x * rstd * gw.x, v.y * rstd * gw.y, v.z * rstd * gw.z, v.w * rstd * gw.w);
            }
        };
#pragma unroll
        for (int j = 0; j < kKept; ++j) {
            const int i = (j * (int)blockDim.x + (int)threadIdx.x) * 4;
            if (i < size) store(i, kept[j]);
        }
        for (int i = (kKept * (int)blockDim.x + (int)threadIdx.x) * 4; i < size; i += (int)blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(src + i), z = load_four<T>(g + i);
            store(i, make_float4(v.x * silu_of<T>(z.x), v.y * silu_of<T>(z.y), v.z * silu_of<T>(z.z), v.w * silu_of<T>(z.w)));
        }
        return;
    }
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float v = src[i] * silu_of<T>(to_f32<T>(g[i]));
        ss += v * v;
    }
    const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + eps);
    for (int i = threadIdx.x; i < size; i += blockDim.x) dst[i] = from_f32<T>(src[i] * silu_of<T>(to_f32<T>(g[i])) * rstd * w[i]);
}

int check_shape(const char* what, const SpaceShape& s, int proj_width, int offset) {
    THN_CHECK_ARG(s.n_heads > 0 && s.vdim > 0 && s.n_state > 0 && s.n_groups > 0 && s.n_heads % s.n_groups == 0 && s.taps > 0,
                  "%s: %d heads of %d in %d groups, state %d, %d taps", what, s.n_heads, s.vdim, s.n_groups, s.n_state, s.taps);
    THN_CHECK_ARG(offset >= 0 && offset + s.channels() <= proj_width, "%s: %d channels from column %d of rows of %d", what,
                  s.channels(), offset, proj_width);
    THN_UNSUPPORTED_IF(s.n_state > 512, "%s: a state of %d, at most 512", what, s.n_state);
    return THN_OK;
}

template <typename T>
void launch_prepare(float* keys, float* values, const void* proj, int proj_width, int offset, const float* conv_w,
                    const float* conv_b, const void* ring, const float* dt_pre, const float* dt_bias, const float* rate,
                    const int* row_slot, const int* row_pos, const int* seq_lens, int n_rows, const SpaceShape& s, cudaStream_t stream) {
    const int kp = padded_keys(s.n_state), vp = padded_values(s.vdim);
    const int items = s.n_heads * (vp / 4) + s.n_groups * 2 * (kp / 4) + s.n_heads;
    const dim3 grid((items + kPrepareThreads - 1) / kPrepareThreads, (n_rows + kRunRows - 1) / kRunRows);
    const uintptr_t piece = 4 * sizeof(T) - 1;
    const int vec = s.vdim % 4 == 0 && s.n_state % 4 == 0 && proj_width % 4 == 0 && offset % 4 == 0 &&
                    (((uintptr_t)proj | (uintptr_t)ring) & piece) == 0;
#define THN_SPACE_PREPARE(K)                                                                                            \
    thn_launch(state_space_prepare_kernel<T, K>, grid, kPrepareThreads, 0, stream, keys, values, (const T*)proj, proj_width, \
               offset, conv_w, conv_b, (const T*)ring, dt_pre, dt_bias, rate, row_slot, row_pos, seq_lens, n_rows, s, kp, vp, vec)
    if (s.taps == 4) THN_SPACE_PREPARE(4);
    else if (s.taps == 3) THN_SPACE_PREPARE(3);
    else if (s.taps == 2) THN_SPACE_PREPARE(2);
    else THN_SPACE_PREPARE(0);
#undef THN_SPACE_PREPARE
}

}  // namespace

// Floats of the scratch that thn_state_space needs for a step of n_rows rows.
THN_API long long thn_state_space_scratch_floats(int n_rows, int n_heads, int vdim, int n_state, int n_groups) {
    return (long long)n_rows * ((long long)n_groups * 2 * padded_keys(n_state) + (long long)n_heads * (padded_values(vdim) + kRecurrenceTail));
}

// y float32 [rows, heads, vdim]; state float32 [slots, heads, vdim, n_state], read and updated; the raw
// inputs [x: heads * vdim | B: groups * n_state | C: groups * n_state] are the columns from `offset` of
// proj [rows, proj_width]; conv_w float32 [channels, taps] (the last tap is the current token's), conv_b
// float32 [channels]; ring [slots, taps, channels] of the activation type (read only: the step's inputs
// go in by thn_conv_ring_update afterwards); dt_pre float32 [rows, heads]; dt_bias, rate (the decay is
// exp(-rate * step)), skip float32 [heads]; seq_lens: the tokens each slot held before the step.
THN_API int thn_state_space(float* y, float* state, float* scratch, const void* proj, int proj_width, int offset,
                            const float* conv_w, const float* conv_b, const void* ring, const float* dt_pre,
                            const float* dt_bias, const float* rate, const float* skip, const int* row_slot,
                            const int* row_pos, const int* seq_lens, const int* cu_seqlens, const int* slots, int n_rows,
                            int n_seqs, int n_heads, int vdim, int n_state, int n_groups, int taps, int dtype,
                            cudaStream_t stream) {
    const SpaceShape s{n_heads, vdim, n_state, n_groups, taps};
    const int bad = check_shape("state_space", s, proj_width, offset);
    if (bad) return bad;
    THN_CHECK_ARG(scratch != nullptr && ((uintptr_t)scratch & 15) == 0 && n_rows >= 0 && n_seqs >= 0, "state_space: scratch missing or unaligned");
    THN_UNSUPPORTED_IF(n_rows > 65535 * kRunRows, "state_space: %d rows", n_rows);
    if (n_rows == 0 || n_seqs == 0) return THN_OK;
    const int kp = padded_keys(n_state), vp = padded_values(vdim);
    float* keys = scratch;
    float* values = scratch + (size_t)n_rows * n_groups * 2 * kp;
    if (dtype == THN_F32)
        launch_prepare<float>(keys, values, proj, proj_width, offset, conv_w, conv_b, ring, dt_pre, dt_bias, rate, row_slot,
                              row_pos, seq_lens, n_rows, s, stream);
    else if (dtype == THN_BF16)
        launch_prepare<__nv_bfloat16>(keys, values, proj, proj_width, offset, conv_w, conv_b, ring, dt_pre, dt_bias, rate,
                                      row_slot, row_pos, seq_lens, n_rows, s, stream);
    else
        THN_CHECK_ARG(false, "state_space: unknown dtype %d", dtype);
    return launch_recurrence(kSteppedDecay, RecurrenceArgs{y, state, keys, 2 * kp, n_groups, values, vp + kRecurrenceTail, skip,
                                                           cu_seqlens, slots, n_seqs, n_heads, n_state, vdim, 1.0f}, stream);
}

// One token per sequence: the same, and the token's raw inputs go into the ring.
THN_API int thn_state_space_decode(float* y, float* state, const void* proj, int proj_width, int offset, const float* conv_w,
                                   const float* conv_b, void* ring, const float* dt_pre, const float* dt_bias,
                                   const float* rate, const float* skip, const int* row_slot, const int* row_pos, int n_rows,
                                   int n_heads, int vdim, int n_state, int n_groups, int taps, int dtype, cudaStream_t stream) {
    const SpaceShape s{n_heads, vdim, n_state, n_groups, taps};
    const int bad = check_shape("state_space_decode", s, proj_width, offset);
    if (bad) return bad;
    const size_t smem = (size_t)(2 * ((n_state + 3) / 4 * 4) + vdim) * sizeof(float);
    THN_UNSUPPORTED_IF(n_rows > 65535 || smem > 48 * 1024, "state_space_decode: %d rows, values of %d", n_rows, vdim);
    if (n_rows <= 0) return THN_OK;
    const dim3 grid(n_heads, n_rows);
    if (dtype == THN_F32)
        thn_launch(state_space_decode_kernel<float>, grid, kDecodeThreads, smem, stream, y, state, (const float*)proj, proj_width,
                   offset, conv_w, conv_b, (float*)ring, dt_pre, dt_bias, rate, skip, row_slot, row_pos, s);
    else if (dtype == THN_BF16)
        thn_launch(state_space_decode_kernel<__nv_bfloat16>, grid, kDecodeThreads, smem, stream, y, state,
                   (const __nv_bfloat16*)proj, proj_width, offset, conv_w, conv_b, (__nv_bfloat16*)ring, dt_pre, dt_bias, rate,
                   skip, row_slot, row_pos, s);
    else
        THN_CHECK_ARG(false, "state_space_decode: unknown dtype %d", dtype);
    return thn_launch_status("state_space_decode");
}

// y float32 [rows, width]; gate of the activation type, rows gate_stride elements apart; gain float32
// [width]; out [rows, width] of the activation type; `parts` equal consecutive parts of a row.
THN_API int thn_gated_group_norm(void* out, const float* y, const void* gate, long long gate_stride, const float* gain,
                                 float eps, int rows, int width, int parts, int dtype, cudaStream_t stream) {
    THN_CHECK_ARG(rows >= 0 && width > 0 && parts > 0 && width % parts == 0 && parts <= 65535 && gate_stride >= width && eps > 0.f,
                  "gated_group_norm: rows of %d in %d parts", width, parts);
    if (rows == 0) return THN_OK;
    const int size = width / parts;
    const size_t element = dtype == THN_BF16 ? 2 : 4;
    const int vec = size % 4 == 0 && gate_stride % 4 == 0 && (((uintptr_t)y | (uintptr_t)gain) & 15) == 0 &&
                    (((uintptr_t)gate | (uintptr_t)out) & (4 * element - 1)) == 0;
    const dim3 grid(rows, parts);
    const int threads = size >= 1024 ? 256 : (size / 4 + 31) / 32 * 32 < 32 ? 32 : (size / 4 + 31) / 32 * 32;
    if (dtype == THN_F32)
        thn_launch(gated_group_norm_kernel<float>, grid, threads, 0, stream, (float*)out, y, (const float*)gate, gate_stride, gain, eps,
                   width, size, vec);
    else if (dtype == THN_BF16)
        thn_launch(gated_group_norm_kernel<__nv_bfloat16>, grid, threads, 0, stream, (__nv_bfloat16*)out, y, (const __nv_bfloat16*)gate,
                   gate_stride, gain, eps, width, size, vec);
    else
        THN_CHECK_ARG(false, "gated_group_norm: unknown dtype %d", dtype);
    return thn_launch_status("gated_group_norm");
}
