// Linear attention with a decayed matrix state: per head a matrix S [key_dim, value_dim], zero at
// a sequence's start, and for every token
//
//     S <- diag(a_t) S + k_t v_t^T          o_t = S^T q_t * q_scale
//
// The decay a_t is one of
//   0  a constant per head (decay[head]); the same for every key channel and token;
//   1  a vector per token and head over the key channels, a = logistic(z)^(1 / tau) with
//      z = gate[row, head * key_dim + d] + gate_bias[head * key_dim + d] (float32), computed as
//      exp(-softplus(-z) / tau).
// q, k and v come from one projected row [q | k | v | ...] of the activation type; with
// silu_inputs they pass silu first.  Everything after the load is float32: the state, the decay
// with its softplus and exponential, the sums.
//
// Other mixers use the same recurrence with other decays and read-outs: linear_attention.cuh.
//
// Two kernels.  linear_attention_prepare does what is the same for every column, once per entry:
// silu of q, k and v where asked, the decay with its softplus and exponential, all to float32 rows
// [row][head][k | q | (decay) | v], the key parts padded with zeros and the values to a multiple of
// 16.  linear_attention_kernel is the recurrence, for every mixer that has one of the kinds of
// linear_attention.cuh.  A column of S (one entry of v and of o) evolves on its own.  16 lanes hold
// COLS neighbouring columns, lane l the key channels 4l .. 4l + 3, 64 + 4l .. of each (runs of four, for
// 16-byte accesses), so that a key, query or decay once loaded serves COLS columns.  One block per
// (sequence, head, 16 columns) walks the sequence's tokens of the step in order.  The tokens come
// through a ring of buffers in shared memory, filled by asynchronous 16-byte copies: a warp copies whole
// tokens, a lane the same pieces of each.  A token's sums over the lanes are not reduced one by one
// (each would be a chain of shuffles that the next token waits behind): every lane leaves its share in
// shared memory, and once a stage of tokens is through, each lane adds up the 16 shares of some
// (token, column) pairs and writes their results.  A row's result depends on its sequence's own
// tokens only, in an order fixed by the sizes.
#include <math.h>

#include "linear_attention.cuh"

namespace {

constexpr int kLanes = kRecurrenceLanes;
constexpr int kColumns = kRecurrenceColumns;  // columns of S per block
constexpr int kGroup = 8;                     // tokens between whose loads no store stands
// tokens per buffer, and buffers: fewer tokens for long keys, so that the ring fits
constexpr int stage_tokens(int per) { return per <= 8 ? 16 : 8; }
constexpr int kBuffers = 3;
// floats between the shares of neighbouring columns: the two column groups of a warp store without bank conflicts
constexpr int share_stride(int cols) { return cols == 2 ? 24 : 20; }

__device__ __forceinline__ void copy16_async(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

// logistic(z)^(1 / tau) = exp(-softplus(-z) / tau), without overflow; in double on the 32-bit path
template <typename T> __device__ __forceinline__ float logistic_power(float z, float inv_tau) {
    const float log_logistic = z >= 0.f ? -log1pf(expf(-z)) : z - log1pf(expf(z));
    return expf(log_logistic * inv_tau);
}
template <> __device__ __forceinline__ float logistic_power<float>(float z, float inv_tau) {
    const double x = (double)z;
    const double log_logistic = x >= 0.0 ? -log1p(exp(-x)) : x - log1p(exp(x));
    return (float)exp(log_logistic * (double)inv_tau);
}

// prepared [rows][heads][parts * kp + vp] float32: k, q (and the decay) over kp entries each, then
// v over vp entries; entries beyond key_dim and value_dim are zero.
template <typename T>
__global__ void linear_attention_prepare_kernel(float* __restrict__ prepared, const T* __restrict__ proj, int proj_width,
                                                int q_offset, int k_offset, int v_offset, const float* __restrict__ gate,
                                                int gate_width, const float* __restrict__ gate_bias, float inv_tau,
                                                long long n, int n_heads, int key_dim, int value_dim, int kp, int vp,
                                                int parts, int silu_inputs) {
    pdl_launch_dependents();
    pdl_wait();
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= n) return;
    const int per_head = parts * kp + vp;
    const long long unit = e / per_head;
    const int c = (int)(e - unit * per_head);
    const long long row = unit / n_heads;
    const int head = (int)(unit - row * n_heads);
    const T* src = proj + row * proj_width;
    float v = 0.f;
    if (c >= parts * kp) {
        const int d = c - parts * kp;
        if (d < value_dim) {
            v = to_f32<T>(src[v_offset + head * value_dim + d]);
            if (silu_inputs) v = silu_of<T>(v);
        }
    } else {
        const int part = c / kp, d = c - part * kp;
        if (d < key_dim) {
            if (part == 2) {
                v = logistic_power<T>(gate[row * gate_width + head * key_dim + d] + (gate_bias ? gate_bias[head * key_dim + d] : 0.f),
                                      inv_tau);
            } else {
                v = to_f32<T>(src[(part == 0 ? k_offset : q_offset) + head * key_dim + d]);
                if (silu_inputs) v = silu_of<T>(v);
            }
        }
    }
    prepared[e] = v;
}

// PER: key channels per lane (a multiple of 4); KP = 16 * PER: the padded key size.  COLS: columns per lane.
template <int PER, int COLS, int KIND>
__global__ void __launch_bounds__(kLanes * kColumns / COLS) linear_attention_kernel(
    float* __restrict__ o, float* __restrict__ state, const float* __restrict__ keys, long long key_stride, int heads_per_unit,
    const float* __restrict__ values, long long value_stride, const float* __restrict__ per_head,
    const int* __restrict__ cu_seqlens, const int* __restrict__ slots, int n_heads, int key_dim, int value_dim, int vp,
    float q_scale) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int KP = kLanes * PER, kStage = stage_tokens(PER), kThreads = kLanes * kColumns / COLS;
    constexpr int PARTS = KIND == kChannelDecay || KIND == kBonusRead ? 3 : 2;     // k, q (and the decay) per token
    constexpr int TAIL = KIND >= kBonusRead ? kRecurrenceTail : 0;
    constexpr int V_AT = PARTS * KP, TAIL_AT = V_AT + kColumns;
    constexpr int ROW = V_AT + kColumns + TAIL;         // floats of one staged token
    constexpr int PIECES = ROW / 4, WARPS = kThreads / 32, PER_LANE = (PIECES + 31) / 32;
    constexpr int SHARE = share_stride(COLS), WARP_COLS = 2 * COLS;
    extern __shared__ __align__(16) float stage_mem[];  // [kBuffers][kStage][ROW], then the shares [kStage][kColumns][SHARE]
    float* shares = stage_mem + (size_t)kBuffers * kStage * ROW;
    const int seq = blockIdx.z, head = blockIdx.y;
    const int col0 = blockIdx.x * kColumns;
    const int lane = threadIdx.x % kLanes, group = threadIdx.x / kLanes;
    const int own_col = col0 + group * COLS;           // this lane's first column
    const int row0 = cu_seqlens[seq], row1 = cu_seqlens[seq + 1];
    if (row0 >= row1) return;
    const int slot = slots[seq];
    float* S = state + ((size_t)slot * n_heads + head) * (size_t)value_dim * key_dim;
    const int unit = head / heads_per_unit, n_units = n_heads / heads_per_unit;
    const size_t key_step = (size_t)n_units * key_stride, value_step = (size_t)n_heads * value_stride;
    const int n_tokens = row1 - row0;
    const int warp = threadIdx.x >> 5, warp_lane = threadIdx.x & 31;

    // a lane's pieces of a token: where each lies in its row, and how far apart rows are
    const float* piece_src[PER_LANE];
    size_t piece_step[PER_LANE];
#pragma unroll
    for (int j = 0; j < PER_LANE; ++j) {
        const int c = (warp_lane + 32 * j) * 4;
        if (c < V_AT) {
            piece_src[j] = keys + ((size_t)row0 * n_units + unit) * key_stride + c;
            piece_step[j] = key_step;
        } else {
            piece_src[j] = values + ((size_t)row0 * n_heads + head) * value_stride +
                           (TAIL != 0 && c >= TAIL_AT ? vp + (c - TAIL_AT) : col0 + (c - V_AT));
            piece_step[j] = value_step;
        }
    }
    auto issue = [&](int stage) {
        const int first = stage * kStage, n = min(kStage, n_tokens - first);
        float* dst = stage_mem + (size_t)(stage % kBuffers) * kStage * ROW + warp_lane * 4;
        for (int t = warp; t < n; t += WARPS) {
#pragma unroll
            for (int j = 0; j < PER_LANE; ++j)
                if (32 * (j + 1) <= PIECES || warp_lane + 32 * j < PIECES)
                    copy16_async(dst + t * ROW + 128 * j, piece_src[j] + (size_t)(first + t) * piece_step[j]);
        }
    };
    const int n_stages = (n_tokens + kStage - 1) / kStage;
#pragma unroll
    for (int i = 0; i < kBuffers - 1; ++i) {
        if (i < n_stages) issue(i);
        copy_commit();
    }

    const bool whole = key_dim % 4 == 0 && ((uintptr_t)state & 15) == 0;
    float s[COLS][PER];
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
        const float* src = S + (size_t)min(own_col + c, value_dim - 1) * key_dim;     // idle columns mirror the last one and store nothing
#pragma unroll
        for (int i = 0; i < PER; i += 4) {
            const int d = (i / 4) * (4 * kLanes) + lane * 4;
            if (whole) {                      // a run of four is inside the key or outside as a whole
                const float4 x = d < key_dim ? *reinterpret_cast<const float4*>(src + d) : make_float4(0.f, 0.f, 0.f, 0.f);
                s[c][i] = x.x; s[c][i + 1] = x.y; s[c][i + 2] = x.z; s[c][i + 3] = x.w;
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j) s[c][i + j] = d + j < key_dim ? src[d + j] : 0.f;
            }
        }
    }
    const float own = per_head != nullptr ? per_head[head] : 0.f;      // the constant decay, or the skip's factor

    // one token: the sums of its read-out over this lane's channels, and the state behind it
    auto advance = [&](const float* tok, float (&sums)[COLS]) {
        float v[COLS];
#pragma unroll
        for (int c = 0; c < COLS; ++c) {
            v[c] = tok[V_AT + group * COLS + c];
            sums[c] = 0.f;
        }
        float decay = own;
        if (KIND == kSteppedDecay) {
            const float2 tail = *reinterpret_cast<const float2*>(tok + TAIL_AT);
            decay = tail.x;
#pragma unroll
            for (int c = 0; c < COLS; ++c) v[c] *= tail.y;
        }
#pragma unroll
        for (int i = 0; i < PER; i += 4) {
            const int d = (i / 4) * (4 * kLanes) + lane * 4;
            const float4 k = *reinterpret_cast<const float4*>(tok + d);
            const float4 q = *reinterpret_cast<const float4*>(tok + KP + d);
            float4 a = make_float4(decay, decay, decay, decay);
            if (PARTS == 3) a = *reinterpret_cast<const float4*>(tok + 2 * KP + d);
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                float* x = s[c] + i;
                if (KIND == kBonusRead) sums[c] += x[0] * q.x + x[1] * q.y + x[2] * q.z + x[3] * q.w;
                x[0] = fmaf(a.x, x[0], k.x * v[c]);      // (one multiply-add links a token's state to the next)
                x[1] = fmaf(a.y, x[1], k.y * v[c]);
                x[2] = fmaf(a.z, x[2], k.z * v[c]);
                x[3] = fmaf(a.w, x[3], k.w * v[c]);
                if (KIND != kBonusRead) sums[c] += x[0] * q.x + x[1] * q.y + x[2] * q.z + x[3] * q.w;
            }
        }
    };
    float* own_share = shares + (size_t)group * COLS * SHARE + lane;

    for (int stage = 0; stage < n_stages; ++stage) {
        copy_wait<kBuffers - 2>();
        __syncthreads();                     // this stage has landed; the buffer of the one before it is free again
        if (stage + kBuffers - 1 < n_stages) issue(stage + kBuffers - 1);
        copy_commit();
        const float* src = stage_mem + (size_t)(stage % kBuffers) * kStage * ROW;
        const int first = stage * kStage, n = min(kStage, n_tokens - first);
        int t0 = 0;
#pragma unroll 1
        for (; t0 + kGroup <= n; t0 += kGroup) {
            float part[kGroup][COLS];
#pragma unroll
            for (int t = 0; t < kGroup; ++t) advance(src + (t0 + t) * ROW, part[t]);
#pragma unroll
            for (int t = 0; t < kGroup; ++t)
#pragma unroll
                for (int c = 0; c < COLS; ++c) own_share[(size_t)((t0 + t) * kColumns + c) * SHARE] = part[t][c];
        }
#pragma unroll 1
        for (; t0 < n; ++t0) {
            float part[COLS];
            advance(src + t0 * ROW, part);
#pragma unroll
            for (int c = 0; c < COLS; ++c) own_share[(size_t)(t0 * kColumns + c) * SHARE] = part[c];
        }
        __syncwarp();
        // the stage's read-outs: this warp's columns, a (token, column) pair per lane and turn
        for (int i = warp_lane; i < n * WARP_COLS; i += 32) {
            const int t = i / WARP_COLS, c = warp * WARP_COLS + i % WARP_COLS;
            const float* share = shares + (size_t)(t * kColumns + c) * SHARE;
            float sum = 0.f;
#pragma unroll
            for (int l = 0; l < kLanes; l += 4) {
                const float4 x = *reinterpret_cast<const float4*>(share + l);
                sum += (x.x + x.y) + (x.z + x.w);
            }
            if (col0 + c < value_dim) {
                const float* tok = src + t * ROW;
                float y = sum * q_scale;
                if (KIND == kBonusRead) y += tok[TAIL_AT] * tok[V_AT + c];
                if (KIND == kSteppedDecay) y += own * tok[V_AT + c];
                o[((size_t)(row0 + first + t) * n_heads + head) * value_dim + col0 + c] = y;
            }
        }
    }
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
        if (own_col + c >= value_dim) break;
        float* dst = S + (size_t)(own_col + c) * key_dim;
#pragma unroll
        for (int i = 0; i < PER; i += 4) {
            const int d = (i / 4) * (4 * kLanes) + lane * 4;
            if (whole) {
                if (d < key_dim) *reinterpret_cast<float4*>(dst + d) = make_float4(s[c][i], s[c][i + 1], s[c][i + 2], s[c][i + 3]);
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (d + j < key_dim) dst[d + j] = s[c][i + j];
            }
        }
    }
}

template <int PER, int COLS, int KIND>
void launch_one(const RecurrenceArgs& a, cudaStream_t stream) {
    constexpr int KP = kLanes * PER, kStage = stage_tokens(PER);
    constexpr int ROW = (KIND == kChannelDecay || KIND == kBonusRead ? 3 : 2) * KP + kColumns + (KIND >= kBonusRead ? kRecurrenceTail : 0);
    const size_t smem = (size_t)kStage * (kBuffers * ROW + kColumns * share_stride(COLS)) * sizeof(float);
    const dim3 grid((a.value_dim + kColumns - 1) / kColumns, a.n_heads, a.n_seqs);
    auto kernel = linear_attention_kernel<PER, COLS, KIND>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    thn_launch_ordered(kernel, grid, kLanes * kColumns / COLS, smem, stream, a.o, a.state, a.keys, a.key_stride, a.n_heads / a.key_units,
                       a.values, a.value_stride, a.per_head, a.cu_seqlens, a.slots, a.n_heads, a.key_dim, a.value_dim,
                       padded_values(a.value_dim), a.q_scale);
}

int g_columns = 0;      // columns per lane for keys up to 128: 1, 2, 4, or 0: the default

template <int PER, int KIND>
void launch_columns(const RecurrenceArgs& a, int columns, cudaStream_t stream) {
    if (columns == 4) launch_one<PER, 4, KIND>(a, stream);
    else if (columns == 2) launch_one<PER, 2, KIND>(a, stream);
    else launch_one<PER, 1, KIND>(a, stream);
}

template <int KIND>
void launch_kind(const RecurrenceArgs& a, cudaStream_t stream) {
    // Four columns a lane load less per multiply-add, two leave twice as many warps: with fewer than 256
    // blocks the latter win (one prompt of 2,048 tokens, 32 heads of 64: 208 against 263 us; four of them 618
    // against 607; 64 heads of 64 over a state of 128: 366 against 364 us, four prompts 1,322 against 1,171).
    const long long blocks = (long long)(padded_values(a.value_dim) / kColumns) * a.n_heads * a.n_seqs;
    const int columns = g_columns ? g_columns : blocks >= 256 ? 4 : 2;
    switch (recurrence_per_lane(a.key_dim)) {
        case 4: return launch_columns<4, KIND>(a, columns, stream);
        case 8: return launch_columns<8, KIND>(a, columns, stream);
        case 16: return launch_one<16, 2, KIND>(a, stream);
        default: return launch_one<32, 1, KIND>(a, stream);
    }
}

template <typename T>
int launch(float* o, float* state, float* prepared, const void* proj, int proj_width, int q_offset, int k_offset, int v_offset,
           const float* decay, const float* gate, int gate_width, const float* gate_bias, float inv_tau,
           const int* cu_seqlens, const int* slots, int n_rows, int n_seqs, int n_heads, int key_dim, int value_dim,
           float q_scale, int mode, int silu_inputs, cudaStream_t stream) {
    const int kp = padded_keys(key_dim), vp = padded_values(value_dim), parts = key_parts(mode), per_head = parts * kp + vp;
    const long long n = (long long)n_rows * n_heads * per_head;
    thn_launch(linear_attention_prepare_kernel<T>, (unsigned)((n + 255) / 256), 256, 0, stream, prepared, (const T*)proj,
               proj_width, q_offset, k_offset, v_offset, gate, gate_width, gate_bias, inv_tau, n, n_heads, key_dim, value_dim, kp,
               vp, parts, silu_inputs);
    return launch_recurrence(mode, RecurrenceArgs{o, state, prepared, per_head, n_heads, prepared + parts * kp, per_head, decay,
                                                  cu_seqlens, slots, n_seqs, n_heads, key_dim, value_dim, q_scale},
                             stream);
}

}  // namespace

// How many columns of S a lane holds, for keys up to 128 (tests and measurement): 1, 2, 4, or 0: the default.
THN_API void thn_set_recurrence_columns(int columns) { g_columns = columns == 1 || columns == 2 || columns == 4 ? columns : 0; }

int launch_recurrence(int kind, const RecurrenceArgs& args, cudaStream_t stream) {
    THN_CHECK_ARG(args.key_units > 0 && args.n_heads % args.key_units == 0, "recurrence: %d heads over %d units of keys",
                  args.n_heads, args.key_units);
    THN_UNSUPPORTED_IF(args.key_dim > 512, "recurrence: keys of %d, at most 512", args.key_dim);
    THN_UNSUPPORTED_IF(args.n_heads > 65535 || args.n_seqs > 65535, "recurrence: %d heads, %d sequences", args.n_heads, args.n_seqs);
    THN_CHECK_ARG((((uintptr_t)args.keys | (uintptr_t)args.values) & 15) == 0 && args.key_stride % 4 == 0 && args.value_stride % 4 == 0,
                  "recurrence: prepared rows are not 16-byte aligned");
    switch (kind) {
        case kConstantDecay: launch_kind<kConstantDecay>(args, stream); break;
        case kChannelDecay: launch_kind<kChannelDecay>(args, stream); break;
        case kBonusRead: launch_kind<kBonusRead>(args, stream); break;
        case kSteppedDecay: launch_kind<kSteppedDecay>(args, stream); break;
        default: THN_CHECK_ARG(false, "recurrence: unknown kind %d", kind);
    }
    return thn_launch_status("recurrence");
}

// Floats of the scratch that thn_linear_attention needs for a step of n_rows rows.
THN_API long long thn_linear_attention_scratch_floats(int n_rows, int n_heads, int key_dim, int value_dim, int mode) {
    return (long long)n_rows * n_heads * ((mode == 1 ? 3 : 2) * (long long)padded_keys(key_dim) + padded_values(value_dim));
}

// o float32 [rows, heads, value_dim]; state float32 [slots, heads, value_dim, key_dim], read and
// updated; proj [rows, proj_width] of the activation type with q, k (heads * key_dim each) and v
// (heads * value_dim) from the given columns; mode 0: decay float32 [heads]; mode 1: gate float32
// [rows, gate_width] (the first heads * key_dim columns), gate_bias float32 [heads * key_dim] or
// null, tau > 0.  The tokens of sequence i are the rows [cu_seqlens[i], cu_seqlens[i + 1]) of the
// step's n_rows rows.  scratch: float32, thn_linear_attention_scratch_floats(...) entries, 16-byte aligned.
THN_API int thn_linear_attention(float* o, float* state, float* scratch, const void* proj, int proj_width, int q_offset, int k_offset,
                                 int v_offset, const float* decay, const float* gate, int gate_width,
                                 const float* gate_bias, float tau, const int* cu_seqlens, const int* slots, int n_rows,
                                 int n_seqs, int n_heads, int key_dim, int value_dim, float q_scale, int mode, int silu_inputs,
                                 int dtype, cudaStream_t stream) {
    THN_CHECK_ARG(n_seqs >= 0 && n_heads > 0 && key_dim > 0 && value_dim > 0, "linear_attention: bad sizes");
    THN_UNSUPPORTED_IF(key_dim > 512, "linear_attention: keys of %d, at most 512", key_dim);
    THN_UNSUPPORTED_IF(n_heads > 65535 || n_seqs > 65535, "linear_attention: %d heads, %d sequences", n_heads, n_seqs);
    THN_CHECK_ARG(mode == 0 ? decay != nullptr : (mode == 1 && gate != nullptr && tau > 0.f && gate_width >= n_heads * key_dim),
                  "linear_attention: decay mode %d without its operands", mode);
    THN_CHECK_ARG(q_offset >= 0 && k_offset >= 0 && v_offset >= 0 && q_offset + n_heads * key_dim <= proj_width &&
                      k_offset + n_heads * key_dim <= proj_width && v_offset + n_heads * value_dim <= proj_width,
                  "linear_attention: q, k, v do not lie inside rows of %d", proj_width);
    THN_CHECK_ARG(scratch != nullptr && ((uintptr_t)scratch & 15) == 0 && n_rows >= 0, "linear_attention: scratch missing or unaligned");
    if (n_seqs == 0 || n_rows == 0) return THN_OK;
    const float inv_tau = mode == 1 ? 1.0f / tau : 0.f;
    if (dtype == THN_F32)
        return launch<float>(o, state, scratch, proj, proj_width, q_offset, k_offset, v_offset, decay, gate, gate_width, gate_bias,
                             inv_tau, cu_seqlens, slots, n_rows, n_seqs, n_heads, key_dim, value_dim, q_scale, mode, silu_inputs,
                             stream);
    if (dtype == THN_BF16)
        return launch<__nv_bfloat16>(o, state, scratch, proj, proj_width, q_offset, k_offset, v_offset, decay, gate, gate_width,
                                     gate_bias, inv_tau, cu_seqlens, slots, n_rows, n_seqs, n_heads, key_dim, value_dim, q_scale,
                                     mode, silu_inputs, stream);
    THN_CHECK_ARG(false, "linear_attention: unknown dtype %d", dtype);
    return THN_OK;
}
