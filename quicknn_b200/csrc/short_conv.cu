// Short causal convolutions over time, one filter per channel, with the last inputs of every sequence as state.
//
//   qnn_causal_conv   v_t = x_t + x_bias;  out_t = sum_j w[:, j] v_(t - taps + 1 + j) + out_bias (+ v_t with `add_input`)
//                     with `act` silu: out_t = silu(that); with `inv`: the first n_heads * head channels are heads, and
//                     inv[t, h] = 1 / sqrt(sum of the squares of head h of out_t, as stored, + inv_eps)
//
// with zeros before a sequence's first position.  A sequence's state is a ring of `taps` rows of C floats: v of position p
// lies in row p mod taps, so a step of any length leaves the rows that it does not replace where they are, and a decode
// step writes a row that no tap of the same step reads.  Prompts, continued sequences and single tokens are one kernel: a
// tap that falls before the step's first row comes from the ring, any other from the step's rows.  Sums are float32 in
// the order of the taps, so they do not depend on how a sequence was cut into steps.
//
// A thread owns VEC channels of `rows` consecutive rows of one sequence; it asks for all of a tile's rows before it uses the
// first.  The threads of a sequence's first tile read the ring (tiles have at least taps - 1 rows) and, after that, write
// the same channels' new rows into it.
#include "common.cuh"

using namespace qnn;

namespace {

constexpr int THREADS = 128;

template <int VEC>
__device__ __forceinline__ void load_v(const void* p, int dt, size_t i, float* o) {
    if (VEC == 8) load8_as_f(p, dt, i, o);
    else o[0] = load_as_f(p, dt, i);
}
// VEC consecutive elements as they lie in memory: loads that do not wait for one another
template <typename T, int VEC> struct Raw {
    static constexpr int PIECES = VEC == 8 ? 8 / Vec16<T>::N : 1;
    Vec16<T> v[PIECES];
    T one;
    __device__ __forceinline__ void load(const T* p) {
        if (VEC == 8) {
#pragma unroll
            for (int i = 0; i < PIECES; ++i) v[i].load(p + i * Vec16<T>::N);
        } else {
            one = *p;
        }
    }
    __device__ __forceinline__ void unpack(float* o) const {
        if (VEC == 8) {
#pragma unroll
            for (int i = 0; i < PIECES; ++i) v[i].unpack(o + i * Vec16<T>::N);
        } else {
            o[0] = to_f(one);
        }
    }
};
template <typename T, int VEC>
__device__ __forceinline__ void store_v(T* p, const float* v) {
    if (VEC == 8) {
#pragma unroll
        for (int i = 0; i < 8 / Vec16<T>::N; ++i) Vec16<T>::store(p + i * Vec16<T>::N, v + i * Vec16<T>::N);
    } else {
        p[0] = from_f<T>(v[0]);
    }
}

// silu of a result that is stored as T: the fast functions where it is rounded to bfloat16
template <typename T> __device__ __forceinline__ float silu_as(float v) { return silu(v); }
template <> __device__ __forceinline__ float silu_as<bf16>(float v) { return activate_fast(v, QNN_ACT_SILU); }

// TAPS > 0: the number of taps and of rows per tile (ROWS) is known here, and the filter and the tile's inputs stay in
// registers; 0: any numbers, inputs are read again for every tap.
template <typename T, int VEC, int TAPS, int ROWS>
__global__ void __launch_bounds__(THREADS)
causal_conv_kernel(const T* __restrict__ x, long long ldx, const void* __restrict__ x_bias, int xb_dt,
                   const void* __restrict__ w, int w_dt, const void* __restrict__ out_bias, int ob_dt, int add_input,
                   T* __restrict__ out, long long ldo, float* state, long long slot_stride, int C, int taps_,
                   const int* __restrict__ seq_row0, const int* __restrict__ seq_len, const int* __restrict__ tok_pos,
                   const int* __restrict__ slots, int rows_, int act, float* __restrict__ inv, int head, int n_heads,
                   float inv_eps) {
    const int taps = TAPS > 0 ? TAPS : taps_, rows = TAPS > 0 ? ROWS : rows_;
    const int b = blockIdx.y;
    // groups of channels; consecutive threads take consecutive groups.  With norms a tile has whole warps, so that the
    // threads of a head are neighbouring lanes.
    const int real = (C + VEC - 1) / VEC, groups = inv != nullptr ? (real + 31) & ~31 : real;
    const unsigned at = blockIdx.x * (unsigned)THREADS + threadIdx.x;
    const int tile = (int)(at / (unsigned)groups), c0 = (int)(at - (unsigned)tile * groups) * VEC;
    const int r0 = tile * rows;                             // first row of this tile within the sequence
    const bool idle = c0 >= C;                              // a lane that only fills a warp up
    float wv[TAPS > 0 ? TAPS : 1][VEC], xb[VEC], ob[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) xb[e] = ob[e] = 0.f;
    // filters and biases are written by no kernel of the step: asked for before the wait for the kernel in front
    if (x_bias != nullptr && !idle) load_v<VEC>(x_bias, xb_dt, c0, xb);
    if (out_bias != nullptr && !idle) load_v<VEC>(out_bias, ob_dt, c0, ob);
    if constexpr (TAPS > 0) {
        float flat[TAPS * VEC];                             // [channel][tap], VEC * TAPS numbers in a row
#pragma unroll
        for (int i = 0; i < TAPS; ++i) load_v<VEC>(w, w_dt, (size_t)(idle ? 0 : c0) * TAPS + i * VEC, flat + i * VEC);
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
            for (int e = 0; e < VEC; ++e) wv[j][e] = flat[e * TAPS + j];
    }
    pdl_wait();
    const int row0 = seq_row0 != nullptr ? seq_row0[b] : b;
    const int n = seq_len != nullptr ? seq_len[b] : 1;
    if (r0 >= n) return;
    const int r1 = min(r0 + rows, n);
    const int slot = slots[b];
    if (slot < 0) {                                         // a row of no sequence
        if (idle) return;
        float z[VEC];
        if (inv != nullptr && c0 < n_heads * head && c0 % head == 0)
            for (int r = r0; r < r1; ++r) inv[(size_t)(row0 + r) * n_heads + c0 / head] = 0.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) z[e] = 0.f;
        for (int r = r0; r < r1; ++r) store_v<T, VEC>(out + (size_t)(row0 + r) * ldo + c0, z);
        return;
    }
    const int first = tok_pos[row0];                        // position of the sequence's first row of this step
    float* ring = state + (size_t)slot * slot_stride + c0;
    // v of row r (may be negative: an earlier step's, or before the sequence)
    auto input = [&](int r, float* v) {
        if (r >= 0) {
            Raw<T, VEC> raw;
            raw.load(x + (size_t)(row0 + r) * ldx + c0);
            raw.unpack(v);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] += xb[e];
        } else if (first + r >= 0) {
            const float* cell = ring + (size_t)((first + r) % taps) * C;
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = cell[e];
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = 0.f;
        }
    };
    if constexpr (TAPS > 0) {
        float v[ROWS + TAPS - 1][VEC];
        if (idle) {
#pragma unroll
            for (int i = 0; i < ROWS + TAPS - 1; ++i)
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[i][e] = 0.f;
        } else if (r0 >= TAPS - 1 && r0 + ROWS <= n) {             // a whole tile with its past among the step's rows: no branches
            Raw<T, VEC> raw[ROWS + TAPS - 1];
#pragma unroll
            for (int i = 0; i < ROWS + TAPS - 1; ++i) raw[i].load(x + (size_t)(row0 + r0 - TAPS + 1 + i) * ldx + c0);
#pragma unroll
            for (int i = 0; i < ROWS + TAPS - 1; ++i) {
                raw[i].unpack(v[i]);
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[i][e] += xb[e];
            }
        } else {
#pragma unroll
            for (int i = 0; i < ROWS + TAPS - 1; ++i) {
                const int r = r0 - TAPS + 1 + i;
                if (r < r1) input(r, v[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            if (r0 + i >= r1) continue;
            float acc[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                acc[e] = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc[e] = fmaf(wv[j][e], v[i + j][e], acc[e]);
                acc[e] += ob[e];
                if (add_input) acc[e] += v[i + TAPS - 1][e];
                if (act) acc[e] = silu_as<T>(acc[e]);
            }
            if (!idle) store_v<T, VEC>(out + (size_t)(row0 + r0 + i) * ldo + c0, acc);
            if (inv != nullptr) {                           // (a warp's rows are one tile's: all its lanes are here)
                float ss = 0.f;
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    const float y = to_f(from_f<T>(acc[e]));
                    ss += y * y;
                }
                for (int o = 1; o < head / VEC; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
                if (!idle && c0 < n_heads * head && c0 % head == 0)
                    inv[(size_t)(row0 + r0 + i) * n_heads + c0 / head] = rsqrtf(ss + inv_eps);
            }
        }
    } else {
        for (int r = r0; r < r1; ++r) {
            float acc[VEC], v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] = v[e] = 0.f;
            for (int j = 0; j < taps; ++j) {
                input(r - taps + 1 + j, v);
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[e] = fmaf(load_as_f(w, w_dt, (size_t)(c0 + e) * taps + j), v[e], acc[e]);
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                acc[e] += ob[e] + (add_input ? v[e] : 0.f);
                if (act) acc[e] = silu_as<T>(acc[e]);
            }
            store_v<T, VEC>(out + (size_t)(row0 + r) * ldo + c0, acc);
        }
    }
    if (r0 == 0 && !idle) {
        for (int r = max(0, n - taps); r < n; ++r) {
            float v[VEC];
            input(r, v);
            float* cell = ring + (size_t)((first + r) % taps) * C;
#pragma unroll
            for (int e = 0; e < VEC; ++e) cell[e] = v[e];
        }
    }
}

// inv[t, h] from rows that are stored already, where the heads' sizes keep them out of the convolution's kernel: a warp per
// (row, head)
template <typename T>
__global__ void inverse_norms_kernel(const T* __restrict__ rows, long long ld, float* __restrict__ inv, int head, int n_heads,
                                     float eps, const int* __restrict__ seq_row0, const int* __restrict__ seq_len,
                                     const int* __restrict__ slots) {
    pdl_wait();
    const int b = blockIdx.y, lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * (THREADS / 32) + (threadIdx.x >> 5);
    const int r = (int)(unit / n_heads), h = (int)(unit - (long long)r * n_heads);
    const int row0 = seq_row0 != nullptr ? seq_row0[b] : b, n = seq_len != nullptr ? seq_len[b] : 1;
    if (r >= n) return;
    const T* at = rows + (size_t)(row0 + r) * ld + (size_t)h * head;
    float ss = 0.f;
    for (int c = lane; c < head; c += 32) {
        const float y = to_f(at[c]);
        ss += y * y;
    }
    ss = warp_sum(ss);
    if (lane == 0) inv[(size_t)(row0 + r) * n_heads + h] = slots[b] >= 0 ? rsqrtf(ss + eps) : 0.f;
}

}  // namespace

// x, out: rows `ldx` / `ldo` elements apart (different buffers).  seq_row0, seq_len (both null: a row per sequence, row b is
// sequence b's next token): the sequences' rows; the position of a sequence's first row is tok_pos of that row.  state: the
// ring of slot s lies at state + s * slot_stride floats.  act: 0 none, 1 silu.  inv (may be null): float32 [rows, n_heads] for
// heads of `head` channels from channel 0 on.
QNN_API int qnn_causal_conv(const void* x, int x_dt, long long ldx, const void* x_bias, int xb_dt, const void* w, int w_dt,
                            const void* out_bias, int ob_dt, int add_input, void* out, int out_dt, long long ldo, float* state,
                            long long slot_stride, int C, int taps, const int* seq_row0, const int* seq_len,
                            const int* tok_pos, const int* slots, int n_seqs, int longest, int act, float* inv, int head,
                            int n_heads, float inv_eps, cudaStream_t st) {
    if (n_seqs <= 0 || longest <= 0) return 0;
    if (C <= 0 || taps < 1 || n_seqs > 65535 || ldx < C || ldo < C || slot_stride < (long long)taps * C) return QNN_ERR_ARGUMENT;
    if (x_dt != out_dt || act < 0 || act > 1) return QNN_ERR_ARGUMENT;
    if (inv != nullptr && (head < 1 || n_heads < 1 || (long long)head * n_heads > C)) return QNN_ERR_ARGUMENT;
    const int xs = x_dt == QNN_DT_BF16 ? 2 : 4, os = xs;
    const bool vec = C % 8 == 0 && (ldx * xs) % 16 == 0 && (ldo * os) % 16 == 0 &&
                     (((uintptr_t)x | (uintptr_t)out | (uintptr_t)x_bias | (uintptr_t)out_bias | (uintptr_t)w) & 15) == 0;
    const bool known = vec && taps >= 2 && taps <= 4;
    int rows = longest > 1 ? 8 : 1;
    if (!known && rows < taps) rows = taps;
    // norms inside the kernel: heads of 1, 2, 4 .. 32 whole eights
    const int lanes = head / 8;
    const bool inside = inv != nullptr && known && head % 8 == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0;
    float* kernel_inv = inside ? inv : nullptr;
    long long groups = (C + (vec ? 7 : 0)) / (vec ? 8 : 1);
    if (inside) groups = (groups + 31) / 32 * 32;
    const long long work = (long long)((longest + rows - 1) / rows) * groups;
    if (work + THREADS > 0xffffffffLL) return QNN_ERR_UNSUPPORTED;
    const dim3 grid((unsigned)((work + THREADS - 1) / THREADS), n_seqs);
#define QNN_CONV_AS(T, V, TP, R)                                                                                       \
    launch_pdl(causal_conv_kernel<T, V, TP, R>, grid, dim3(THREADS), 0, st, (const T*)x, ldx, x_bias, xb_dt, w, w_dt,   \
               out_bias, ob_dt, add_input, (T*)out, ldo, state, slot_stride, C, taps, seq_row0, seq_len, tok_pos, slots, rows,     \
               act, kernel_inv, head, n_heads, inv_eps)
#define QNN_CONV(V, TP, R)                                        \
    do {                                                          \
        if (x_dt == QNN_DT_BF16) QNN_CONV_AS(bf16, V, TP, R);     \
        else QNN_CONV_AS(float, V, TP, R);                        \
    } while (0)
#define QNN_CONV_TAPS(R)               \
    if (taps == 4) QNN_CONV(8, 4, R);  \
    else if (taps == 3) QNN_CONV(8, 3, R); \
    else QNN_CONV(8, 2, R);
    if (known && rows == 8) { QNN_CONV_TAPS(8) }
    else if (known) { QNN_CONV_TAPS(1) }
    else if (vec) QNN_CONV(8, 0, 1);
    else QNN_CONV(1, 0, 1);
#undef QNN_CONV_TAPS
#undef QNN_CONV
#undef QNN_CONV_AS
    if (inv != nullptr && !inside) {
        const dim3 g2((unsigned)(((long long)longest * n_heads + THREADS / 32 - 1) / (THREADS / 32)), n_seqs);
        if (x_dt == QNN_DT_BF16)
            launch_pdl(inverse_norms_kernel<bf16>, g2, dim3(THREADS), 0, st, (const bf16*)out, ldo, inv, head, n_heads, inv_eps,
                       seq_row0, seq_len, slots);
        else
            launch_pdl(inverse_norms_kernel<float>, g2, dim3(THREADS), 0, st, (const float*)out, ldo, inv, head, n_heads,
                       inv_eps, seq_row0, seq_len, slots);
    }
    QNN_LAUNCH_CHECK();
}
