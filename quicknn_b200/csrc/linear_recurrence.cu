// The real-gated linear recurrence (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient
// Language Models"): one number of state per channel.
//
//   r = sigmoid(zr + br),  i = sigmoid(zi + bi),  log a = -decay * r,  a = exp(log a)
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u_t            out = scale * S_t * gelu(y_t + by)
//
// `decay` (one positive number per channel) is formed when the model is loaded.  Everything from the gates' logits to the
// state is float32; 1 - a^2 is formed as -expm1(2 log a), which keeps its digits where a is near 1.
//
// A thread walks one channel of one sequence.  Sequences of more than one segment (of 32 rows) are walked in segments side by
// side, since the recurrence is linear in S: first (a, the added term) take the place of the gates' logits and every segment
// leaves the product of its a and the state that it reaches from 0 (the first segment: from the sequence's state); then
// every segment's starting state follows from those in order (inside the last kernel; with many segments in one of its own)
// and the segments are walked again with the output.  The last segment's thread leaves the state.
//
//   qnn_recurrence_gates    bfloat16 rows: the gates' block-diagonal product and the first of these passes in one kernel.  A CTA
//                           forms the r and i logits of 64 channels for 128 rows (mma.sync m16n8k16, a cp.async ring), leaves
//                           them in shared memory, and its threads, one per channel and segment, turn them into (a, term).
//   qnn_linear_recurrence   the passes (all of them, or what follows qnn_recurrence_gates)
#include "common.cuh"

using namespace qnn;

namespace {

constexpr int THREADS = 128;
constexpr int INLINE_PREFIX = 8;        // segments up to which a segment forms its own starting state

struct Rec {
    float* z;                   // logits [rows][ldz]: channel c of block b = c / part: columns 2 b part + (c - b part), + part for i
    const void* rb;             // biases [C]
    const void* ib;
    const float* decay;         // [C]
    const void* u;              // rows of pitch ldu
    const void* y;              // rows of pitch ldy, may be null (no output gate): out = scale * S
    const void* yb;             // [C] or null
    void* out;                  // rows of pitch ldo
    float* state;               // slot s: state + s * slot_stride, [C]
    float* scratch;             // [sequences][segments][3][C]: product of a (later: the starting state), state reached,
                                // (segment 0:) the state it began with
    const int* seq_row0;
    const int* seq_len;
    const int* slots;
    long long ldz, ldu, ldy, ldo, slot_stride;
    int b_dt, yb_dt, C, part, seg, nseg, prefixed;
    float scale;
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// (a, what is added to the state) of a row and channel
__device__ __forceinline__ float2 gates(float zr, float zi, float br, float bi, float decay, float u) {
    const float la = -decay * sigmoid_f(zr + br);
    return make_float2(expf(la), sqrtf(-expm1f(2.f * la)) * sigmoid_f(zi + bi) * u);
}

template <bool AGGREGATE, typename T>       // T: of u, y and out; AGGREGATE: the first of the two
// kernels; else with nseg > 1 the second, with nseg 1 the only one
__global__ void __launch_bounds__(THREADS) recurrence_kernel(const Rec p) {
    pdl_wait();
    const int c = blockIdx.x * THREADS + threadIdx.x;
    if (c >= p.C) return;
    const int b = blockIdx.z, sg = blockIdx.y;
    const int row0 = p.seq_row0 != nullptr ? p.seq_row0[b] : b;
    const int n = p.seq_len != nullptr ? p.seq_len[b] : 1;
    const int slot = p.slots[b];
    const int r0 = sg * p.seg, r1 = min(r0 + p.seg, n);
    if (r0 >= n) return;
    const T* up = (const T*)p.u;
    const T* yp = (const T*)p.y;
    T* op = (T*)p.out;
    if (slot < 0) {
        if (!AGGREGATE)
            for (int r = r0; r < r1; ++r) op[(size_t)(row0 + r) * p.ldo + c] = from_f<T>(0.f);
        return;
    }
    const int blk = c / p.part;
    const size_t zc = (size_t)blk * 2 * p.part + (c - blk * p.part);
    float* state = p.state + (size_t)slot * p.slot_stride + c;
    const float br = load_as_f(p.rb, p.b_dt, c), bi = load_as_f(p.ib, p.b_dt, c), decay = p.decay[c];
    if (AGGREGATE) {
        float* sc = p.scratch + ((size_t)b * p.nseg + sg) * 3 * p.C + c;
        float S = 0.f, all = 1.f;
        if (sg == 0) {
            S = *state;
            sc[2 * (size_t)p.C] = S;
        }
#pragma unroll 4
        for (int r = r0; r < r1; ++r) {
            float* z = p.z + (size_t)(row0 + r) * p.ldz + zc;
            const float2 ab = gates(z[0], z[p.part], br, bi, decay, to_f(up[(size_t)(row0 + r) * p.ldu + c]));
            z[0] = ab.x;
            z[p.part] = ab.y;
            all *= ab.x;
            S = fmaf(ab.x, S, ab.y);
        }
        sc[0] = all;
        sc[p.C] = S;
        return;
    }
    const bool whole = p.nseg == 1;
    float S;
    if (whole) {
        S = *state;
    } else {
        const float* sc = p.scratch + (size_t)b * p.nseg * 3 * p.C + c;
        if (p.prefixed) {
            S = sc[(size_t)sg * 3 * p.C];
        } else {
            S = sg == 0 ? sc[2 * (size_t)p.C] : sc[p.C];
#pragma unroll 4
            for (int k = 1; k < sg; ++k) S = fmaf(sc[(size_t)k * 3 * p.C], S, sc[((size_t)k * 3 + 1) * p.C]);
        }
    }
    const float yb = p.yb != nullptr ? load_as_f(p.yb, p.yb_dt, c) : 0.f;
    constexpr int AHEAD = 8;                                   // rows asked for together
    for (int r = r0; r < r1; r += AHEAD) {
        float za[AHEAD], zb[AHEAD];
        T yv[AHEAD], uv[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const size_t row = (size_t)(row0 + min(r + i, r1 - 1));
            za[i] = p.z[row * p.ldz + zc];
            zb[i] = p.z[row * p.ldz + zc + p.part];
            if (yp != nullptr) yv[i] = yp[row * p.ldy + c];
            if (whole) uv[i] = up[row * p.ldu + c];
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (r + i >= r1) continue;
            float2 ab = make_float2(za[i], zb[i]);
            if (whole) ab = gates(ab.x, ab.y, br, bi, decay, to_f(uv[i]));
            S = fmaf(ab.x, S, ab.y);
            const float gate = yp == nullptr ? 1.f : (sizeof(T) == 2 ? activate_fast(to_f(yv[i]) + yb, QNN_ACT_GELU_TANH) : gelu_tanh(to_f(yv[i]) + yb));
            op[(size_t)(row0 + r + i) * p.ldo + c] = from_f<T>(p.scale * S * gate);
        }
    }
    if (r1 == n) *state = S;
}

// Every segment's starting state in the place of its product of a: a thread per channel walks the segments in order.
__global__ void __launch_bounds__(THREADS) recurrence_prefix_kernel(const Rec p) {
    pdl_wait();
    const int c = blockIdx.x * THREADS + threadIdx.x, b = blockIdx.y;
    if (c >= p.C || p.slots[b] < 0) return;
    const int n = p.seq_len != nullptr ? p.seq_len[b] : 1;
    const int segs = (n + p.seg - 1) / p.seg;
    float* sc = p.scratch + (size_t)b * p.nseg * 3 * p.C + c;
    float S = sc[2 * (size_t)p.C];
    constexpr int AHEAD = 16;
    for (int k = 0; k < segs; k += AHEAD) {
        float all[AHEAD], reached[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const int kk = min(k + i, segs - 1);
            all[i] = sc[(size_t)kk * 3 * p.C];
            reached[i] = sc[((size_t)kk * 3 + 1) * p.C];
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (k + i >= segs) continue;
            sc[(size_t)(k + i) * 3 * p.C] = S;
            S = k + i == 0 ? reached[i] : fmaf(all[i], S, reached[i]);
        }
    }
}

}  // namespace

// seq_row0, seq_len both null: a row per sequence.  `longest`: the most rows that one sequence brings.  With nseg > 1
// (segments of `seg` rows) z is overwritten and scratch holds n_seqs * nseg * 3 * C floats; gates_done: both are what
// qnn_recurrence_gates left.
QNN_API int qnn_linear_recurrence(float* z, long long ldz, const void* rb, const void* ib, int b_dt, const float* decay,
                                  const void* u, int u_dt, long long ldu, const void* y, int y_dt, long long ldy,
                                  const void* yb, int yb_dt, float scale, void* out, int out_dt, long long ldo, float* state,
                                  long long slot_stride, const int* seq_row0, const int* seq_len, const int* slots, int n_seqs,
                                  int C, int part, int seg, int nseg, float* scratch, int gates_done,
                                  cudaStream_t st) {
    if (n_seqs <= 0) return 0;
    if (u_dt != out_dt || (y != nullptr && y_dt != u_dt)) return QNN_ERR_ARGUMENT;
    if (C <= 0 || part <= 0 || C % part || nseg < 1 || seg < 1 || n_seqs > 65535 || nseg > 65535 || ldz < 2LL * C ||
        ldu < C || ldo < C || (y != nullptr && ldy < C) || slot_stride < C || (nseg > 1 && (scratch == nullptr || seq_row0 == nullptr)))
        return QNN_ERR_ARGUMENT;
    Rec p;
    p.z = z; p.rb = rb; p.ib = ib; p.decay = decay; p.u = u; p.y = y; p.yb = yb; p.out = out; p.state = state;
    p.scratch = scratch; p.seq_row0 = seq_row0; p.seq_len = seq_len; p.slots = slots; p.ldz = ldz; p.ldu = ldu; p.ldy = ldy;
    p.ldo = ldo; p.slot_stride = slot_stride; p.b_dt = b_dt; p.yb_dt = yb_dt;
    p.C = C; p.part = part; p.seg = seg; p.nseg = nseg; p.scale = scale;
    p.prefixed = nseg > INLINE_PREFIX ? 1 : 0;
    const dim3 grid((C + THREADS - 1) / THREADS, nseg, n_seqs);
    if (nseg > 1 && !gates_done) {
        launch_pdl(u_dt == QNN_DT_BF16 ? recurrence_kernel<true, bf16> : recurrence_kernel<true, float>, grid, dim3(THREADS), 0, st, p);
        const cudaError_t e = cudaGetLastError();
        if (e != cudaSuccess) return (int)e;
    }
    if (p.prefixed) {
        launch_pdl(recurrence_prefix_kernel, dim3(grid.x, n_seqs), dim3(THREADS), 0, st, p);
        const cudaError_t e = cudaGetLastError();
        if (e != cudaSuccess) return (int)e;
    }
    launch_pdl(u_dt == QNN_DT_BF16 ? recurrence_kernel<false, bf16> : recurrence_kernel<false, float>, grid, dim3(THREADS), 0, st, p);
    QNN_LAUNCH_CHECK();
}
