// The recurrence over a decayed matrix state that several mixers share (linear_attention.cu holds
// the kernel).  Per head a matrix S [key_dim, value_dim]; per token a key, a query, a value:
//
//   kConstantDecay    S <- a_h S + k v^T            o = S^T q * q_scale        a_h = per_head[h]
//   kChannelDecay     S <- diag(a) S + k v^T        o = S^T q * q_scale        a staged with the token
//   kBonusRead        o = S^T q + b v               S <- diag(a) S + k v^T     (the read-out sees the state
//                     before the token; b, the token's own share, is staged with it)
//   kSteppedDecay     S <- a S + k (t v)^T          o = S^T q + per_head[h] v  (one decay a and one step size t
//                     per token and head, staged with it)
//
// The operands are float32 rows that a prepare kernel of the mixer has written.  Keys: per row and
// unit (a unit is a head, or a group of neighbouring heads that share keys and queries)
// [k | q | (a)], each part padded with zeros to padded_keys(key_dim) floats.  Values: per row and
// head [v], padded to padded_values(value_dim), then for the last two kinds a tail of four floats:
// (b, -, -, -) or (a, t, -, -).
#pragma once

#include "common.cuh"

enum RecurrenceKind { kConstantDecay = 0, kChannelDecay = 1, kBonusRead = 2, kSteppedDecay = 3 };

constexpr int kRecurrenceLanes = 16;       // lanes that hold a column of S
constexpr int kRecurrenceColumns = 16;     // columns of S per block
constexpr int kRecurrenceTail = 4;

// key channels per lane: runs of four
inline int recurrence_per_lane(int key_dim) { return key_dim <= 64 ? 4 : key_dim <= 128 ? 8 : key_dim <= 256 ? 16 : 32; }
inline int padded_keys(int key_dim) { return kRecurrenceLanes * recurrence_per_lane(key_dim); }
inline int padded_values(int value_dim) { return (value_dim + kRecurrenceColumns - 1) / kRecurrenceColumns * kRecurrenceColumns; }
inline int key_parts(int kind) { return kind == kChannelDecay || kind == kBonusRead ? 3 : 2; }
inline int value_tail(int kind) { return kind >= kBonusRead ? kRecurrenceTail : 0; }

struct RecurrenceArgs {
    float* o;                 // [rows, heads, value_dim]
    float* state;             // [slots, heads, value_dim, key_dim], read and updated
    const float* keys;        // rows of key_units units, key_stride floats each
    long long key_stride;
    int key_units;            // a divisor of n_heads
    const float* values;      // rows of heads, value_stride floats each
    long long value_stride;
    const float* per_head;    // see the kinds above
    const int* cu_seqlens;
    const int* slots;
    int n_seqs, n_heads, key_dim, value_dim;
    float q_scale;
};

int launch_recurrence(int kind, const RecurrenceArgs& args, cudaStream_t stream);
