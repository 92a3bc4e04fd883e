// The gated delta rule: a matrix state S [dim, vdim] per (sequence, head) that decays, is asked what the key finds in it, and
// gets the difference to the value written at that key.
//
//   S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t            float32
//   beta_t = sigmoid(b_t),   g_t = exp(-exp(A) softplus(a_t + bias))                              one of each per value head
//
// k_t and q_t are unit vectors times a constant: rows hold the vectors as they come out of the convolution and an array holds
// 1 / length per (row, head) (qnn_causal_conv with `inv`); the product is formed in float32 where the rows are read, so it is
// never rounded.  n_kv query/key heads serve n_heads value heads.
//
//   qnn_delta_chunks   per chunk of 16 rows and value head: what does not depend on the state
//   qnn_delta_scan     walks the chunks of every sequence in order, from the slot's state and back into it
//   qnn_delta_step     one token per sequence, everything between the input product and the output product in one kernel
//
// Chunks (Yang et al., "Parallelizing Linear Transformers with the Delta Rule over Sequence Length").  With S the state before a
// chunk, P_t the product of g_1 .. g_t and D_ti the product of g_(i+1) .. g_t,
//
//   u_t + sum_(i<t) beta_t D_ti (k_i . k_t) u_i = beta_t (v_t - P_t S^T k_t)           (I + L) U = diag(beta) (V - P K S)
//   o_t = P_t S^T q_t + sum_(i<=t) D_ti (k_i . q_t) u_i                                 O = P Q S + A U
//   S'  = P_16 S + sum_t D_16,t k_t u_t^T
//
// qnn_delta_chunks forms T = (I + L)^-1 diag(beta), A, P and D_16,. by products of decays, never by their logarithms' differences.
// Every decay product is at most 1.  The scan is then three small matrix products per chunk instead of 16 steps that wait for
// one another.  The order of the sums depends on the sizes only; where a sequence's chunks start moves results by rounding.
#include "common.cuh"

using namespace qnn;

namespace {

constexpr int CK = 16;                       // rows of a chunk
constexpr int RECORD = 2 * CK * CK + 2 * CK; // floats that qnn_delta_chunks leaves per (chunk, value head): T, A, P, D
constexpr int MAX_DIM = 256;

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float beta_of(float b) { return 1.f / (1.f + expf(-b)); }
__device__ __forceinline__ float decay_of(float a, float rate, float bias) { return expf(-rate * softplus(a + bias)); }

// chunk c of sequence b is record slot (row0 / 16 + b + c): the slots of different sequences never meet, and T / 16 + B of
// them hold a step's chunks whatever its sequences' lengths
__device__ __forceinline__ size_t record_of(int row0, int b, int c) { return (size_t)(row0 / CK + b + c); }

template <typename T>
__global__ void __launch_bounds__(128)
delta_chunks_kernel(const T* __restrict__ q, const T* __restrict__ k, long long ld, const float* __restrict__ inv, int ldi,
                    const float* __restrict__ pre, int ldp, const float* __restrict__ rate, const float* __restrict__ bias,
                    float q_scale, const int* __restrict__ seq_row0, const int* __restrict__ seq_len, float* __restrict__ rec,
                    int H, int G, int dim) {
    extern __shared__ __align__(16) float sm[];
    const int pitch = ((dim + 3) & ~3) + 4;                   // rows on 16 bytes, four banks apart
    float* ks = sm;                                           // [CK][pitch]
    float* qs = ks + CK * pitch;
    float* kk = qs + CK * pitch;                              // [CK][CK + 1]: k_t . k_j
    float* qk = kk + CK * (CK + 1);                           // q_t . k_j
    float* low = qk + CK * (CK + 1);                          // [4 warps][CK][CK + 1]
    pdl_wait();
    const int c = blockIdx.x, g = blockIdx.y, b = blockIdx.z;
    const int n = seq_len != nullptr ? seq_len[b] : 1, row0 = seq_row0 != nullptr ? seq_row0[b] : b, t0 = c * CK;
    if (t0 >= n) return;
    const int nt = min(CK, n - t0);
    const int dpad = pitch - 4;
    for (int i = threadIdx.x; i < CK * dpad; i += 128) {
        const int t = i / dpad, d = i - t * dpad;
        float kv = 0.f, qv = 0.f;
        if (t < nt && d < dim) {
            const size_t row = (size_t)(row0 + t0 + t);
            const float iq = inv[row * ldi + g] * q_scale, ik = inv[row * ldi + G + g];
            qv = to_f(q[row * ld + (size_t)g * dim + d]) * iq;
            kv = to_f(k[row * ld + (size_t)g * dim + d]) * ik;
        }
        ks[t * pitch + d] = kv;
        qs[t * pitch + d] = qv;
    }
    __syncthreads();
    {   // a thread forms row t of both products at columns j and j + 8
        const int t = threadIdx.x >> 3, j = threadIdx.x & 7;
        float kk0 = 0.f, kk1 = 0.f, qk0 = 0.f, qk1 = 0.f;
        for (int d = 0; d < dpad; d += 4) {
            const float4 a = *reinterpret_cast<const float4*>(ks + t * pitch + d), e = *reinterpret_cast<const float4*>(qs + t * pitch + d);
            const float4 x = *reinterpret_cast<const float4*>(ks + j * pitch + d), y = *reinterpret_cast<const float4*>(ks + (j + 8) * pitch + d);
            kk0 += a.x * x.x + a.y * x.y + a.z * x.z + a.w * x.w;
            kk1 += a.x * y.x + a.y * y.y + a.z * y.z + a.w * y.w;
            qk0 += e.x * x.x + e.y * x.y + e.z * x.z + e.w * x.w;
            qk1 += e.x * y.x + e.y * y.y + e.z * y.z + e.w * y.w;
        }
        kk[t * (CK + 1) + j] = kk0;
        kk[t * (CK + 1) + j + 8] = kk1;
        qk[t * (CK + 1) + j] = qk0;
        qk[t * (CK + 1) + j + 8] = qk1;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, j = lane & (CK - 1);
    float* L = low + warp * CK * (CK + 1);
    const int per = H / G;
    for (int s = warp; s < per; s += 4) {
        const int h = g * per + s;
        float* out = rec + (record_of(row0, b, c) * H + h) * RECORD;
        float be = 0.f, ga = 1.f;                             // of row j; rows beyond the sequence write nothing and decay nothing
        if (j < nt) {
            const float* pr = pre + (size_t)(row0 + t0 + j) * ldp;
            be = beta_of(pr[h]);
            ga = decay_of(pr[H + h], rate[h], bias[h]);
        }
        // lanes 0..15: column j of L; lanes 16..31: column j of A.  d runs through D_tj.
        float d = 1.f, p = 1.f;
#pragma unroll
        for (int t = 0; t < CK; ++t) {
            const float gt = __shfl_sync(0xffffffffu, ga, t), bt = __shfl_sync(0xffffffffu, be, t);
            if (t > j) d *= gt;
            p *= gt;
            if (lane < CK) {
                L[t * (CK + 1) + j] = t > j ? bt * d * kk[t * (CK + 1) + j] : 0.f;
                if (t == j) out[2 * CK * CK + t] = p;
            } else {
                out[CK * CK + t * CK + j] = t >= j ? d * qk[t * (CK + 1) + j] : 0.f;
            }
        }
        if (lane < CK) out[2 * CK * CK + CK + j] = d;
        __syncwarp();
        if (lane < CK) {                                      // column j of (I + L)^-1, from the top
            float x[CK];
#pragma unroll
            for (int t = 0; t < CK; ++t) {
                float s0 = t == j ? 1.f : 0.f;
#pragma unroll
                for (int i = 0; i < t; ++i) s0 -= L[t * (CK + 1) + i] * x[i];
                x[t] = s0;
                out[t * CK + j] = s0 * be;
            }
        }
        __syncwarp();
    }
}

// ---- the scan ---------------------------------------------------------------------------------------------------
// A block owns 16 * CPT value columns of one (sequence, head).  Eight lanes share a group of CPT columns, each with an eighth
// of the key channels of the state in registers (RPT of them); a warp has four groups, and everything of a chunk but the
// staging happens inside a warp: the products of the state with the chunk's keys and queries (partial sums of four rows and
// columns at a time, summed over the eight lanes by a reduction that leaves one sum per lane), the two 16 x 16 products per
// column, the state's update.
constexpr int SHARE = 8, SCAN_THREADS = 128, GROUPS = SCAN_THREADS / SHARE;
constexpr int MAT = CK + 4;                  // pitch of T and A in shared memory

template <int RPT, int CPT>
struct ScanBuf {
    static constexpr int COLS = GROUPS * CPT, PART = RPT + 4, ROW = SHARE * PART;
    static constexpr int K = 0, Q = K + CK * ROW, V = Q + CK * ROW, T = V + CK * COLS, A = T + CK * MAT, P = A + CK * MAT,
                         D = P + CK, FLOATS = D + CK;
    static constexpr int WCOLS = 4 * CPT;    // columns of a warp
    static constexpr int WORK = 3 * CK * WCOLS;                // per warp: K S, Q S, then X and U
    static constexpr size_t bytes(int buffers) { return ((size_t)buffers * FLOATS + 4 * WORK) * sizeof(float); }
};

template <typename T, int RPT, int CPT, bool VEC>
__global__ void __launch_bounds__(SCAN_THREADS)
delta_scan_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long long ld,
                  const float* __restrict__ inv, int ldi, float q_scale, const float* __restrict__ rec,
                  const int* __restrict__ seq_row0, const int* __restrict__ seq_len, const int* __restrict__ slots,
                  float* __restrict__ state, long long slot_stride, float* __restrict__ out, long long ldo, int H, int G, int dim,
                  int vdim) {
    using B = ScanBuf<RPT, CPT>;
    constexpr int DIMP = RPT * SHARE, COLS = B::COLS;
    constexpr bool AHEAD = RPT <= 16;                         // two buffers, the next chunk's loads in registers meanwhile
    constexpr int N8 = CK * DIMP / 8 / SCAN_THREADS > 0 ? CK * DIMP / 8 / SCAN_THREADS : 1;        // eights of K per thread
    extern __shared__ __align__(16) float sm[];
    const int h = blockIdx.y, c0 = blockIdx.x * COLS, b = blockIdx.z;
    pdl_wait();
    const int n = seq_len != nullptr ? seq_len[b] : 1, row0 = seq_row0 != nullptr ? seq_row0[b] : b, slot = slots[b];
    if (n <= 0) return;
    if (slot < 0) {                                           // rows of no sequence
        const int live = min(COLS, vdim - c0);
        for (int i = threadIdx.x; i < n * live; i += SCAN_THREADS)
            out[(size_t)(row0 + i / live) * ldo + (size_t)h * vdim + c0 + i % live] = 0.f;
        return;
    }
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, part = lane & (SHARE - 1), grp = tid / SHARE;
    const int col = c0 + grp * CPT;
    const int g = h / (H / G);
    float* my_state = state + (size_t)slot * slot_stride + ((size_t)h * dim) * vdim + col;
    float S[RPT][CPT];
#pragma unroll
    for (int r = 0; r < RPT; ++r)
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const int i = part * RPT + r;
            S[r][c] = (i < dim && col + c < vdim) ? my_state[(size_t)i * vdim + c] : 0.f;
        }
    float* work = sm + (AHEAD ? 2 : 1) * B::FLOATS + warp * B::WORK;
    float* wk = work;                                         // [CK][WCOLS] K S, then V - P K S
    float* wq = work + CK * B::WCOLS;                         // [CK][WCOLS] Q S
    float* wu = work + 2 * CK * B::WCOLS;                     // [CK][WCOLS] U
    // what is loaded stays as it came until `put`: the loads are in flight while the chunk before is walked
    constexpr int PIECES = VEC ? 8 / Vec16<T>::N : 1;
    Vec16<T> rq[VEC ? N8 : 1][PIECES], rk[VEC ? N8 : 1][PIECES], rv[PIECES];
    T sq[VEC ? 1 : N8 * 8], sk[VEC ? 1 : N8 * 8], sv[VEC ? 1 : CK * COLS / SCAN_THREADS];
    float iq[N8 * (VEC ? 1 : 8)], ik[N8 * (VEC ? 1 : 8)];
    float4 rm[2];
    constexpr int VT = CK * COLS / 8;                         // threads that fetch eight values each
    auto fetch = [&](int t0) {
        const int nt = min(CK, n - t0);
        if constexpr (VEC) {
#pragma unroll
            for (int e = 0; e < N8; ++e) {
                const int i = tid + e * SCAN_THREADS, t = i / (DIMP / 8), d = (i - t * (DIMP / 8)) * 8;
                iq[e] = ik[e] = 0.f;
#pragma unroll
                for (int p = 0; p < PIECES; ++p) { rq[e][p].zero(); rk[e][p].zero(); }
                if (t < nt && d < dim) {
                    const size_t row = (size_t)(row0 + t0 + t);
#pragma unroll
                    for (int p = 0; p < PIECES; ++p) {
                        rq[e][p].load(q + row * ld + (size_t)g * dim + d + p * Vec16<T>::N);
                        rk[e][p].load(k + row * ld + (size_t)g * dim + d + p * Vec16<T>::N);
                    }
                    iq[e] = inv[row * ldi + g];
                    ik[e] = inv[row * ldi + G + g];
                }
            }
            if (tid < VT) {
                const int t = tid / (COLS / 8), c = (tid - t * (COLS / 8)) * 8;
#pragma unroll
                for (int p = 0; p < PIECES; ++p) rv[p].zero();
                if (t < nt && c0 + c < vdim)
#pragma unroll
                    for (int p = 0; p < PIECES; ++p)
                        rv[p].load(v + (size_t)(row0 + t0 + t) * ld + (size_t)h * vdim + c0 + c + p * Vec16<T>::N);
            }
        } else {
#pragma unroll
            for (int e = 0; e < N8 * 8; ++e) {
                const int i = tid + e * SCAN_THREADS, t = i / DIMP, d = i - t * DIMP;
                sq[e] = sk[e] = from_f<T>(0.f);
                iq[e] = ik[e] = 0.f;
                if (t < nt && d < dim) {
                    const size_t row = (size_t)(row0 + t0 + t);
                    sq[e] = q[row * ld + (size_t)g * dim + d];
                    sk[e] = k[row * ld + (size_t)g * dim + d];
                    iq[e] = inv[row * ldi + g];
                    ik[e] = inv[row * ldi + G + g];
                }
            }
#pragma unroll
            for (int e = 0; e < CK * COLS / SCAN_THREADS; ++e) {
                const int i = tid + e * SCAN_THREADS, t = i / COLS, c = i - t * COLS;
                sv[e] = (t < nt && c0 + c < vdim) ? v[(size_t)(row0 + t0 + t) * ld + (size_t)h * vdim + c0 + c] : from_f<T>(0.f);
            }
        }
        const float4* m = reinterpret_cast<const float4*>(rec + (record_of(row0, b, t0 / CK) * H + h) * RECORD);
        rm[0] = m[tid];
        if (tid < RECORD / 4 - SCAN_THREADS) rm[1] = m[SCAN_THREADS + tid];
    };
    auto put = [&](float* buf) {
        if constexpr (VEC) {
#pragma unroll
            for (int e = 0; e < N8; ++e) {
                const int i = tid + e * SCAN_THREADS, t = i / (DIMP / 8), d = (i - t * (DIMP / 8)) * 8;
                if (t < CK) {
                    float fq[8], fk[8];
#pragma unroll
                    for (int p = 0; p < PIECES; ++p) {
                        rq[e][p].unpack(fq + p * Vec16<T>::N);
                        rk[e][p].unpack(fk + p * Vec16<T>::N);
                    }
                    const float a = iq[e] * q_scale;
#pragma unroll
                    for (int u = 0; u < 8; ++u) { fq[u] *= a; fk[u] *= ik[e]; }
#pragma unroll
                    for (int u = 0; u < 8; u += 4) {
                        const int at = t * B::ROW + ((d + u) / RPT) * B::PART + (d + u) % RPT;
                        *reinterpret_cast<float4*>(buf + B::Q + at) = make_float4(fq[u], fq[u + 1], fq[u + 2], fq[u + 3]);
                        *reinterpret_cast<float4*>(buf + B::K + at) = make_float4(fk[u], fk[u + 1], fk[u + 2], fk[u + 3]);
                    }
                }
            }
            if (tid < VT) {
                float f[8];
#pragma unroll
                for (int p = 0; p < PIECES; ++p) rv[p].unpack(f + p * Vec16<T>::N);
#pragma unroll
                for (int u = 0; u < 8; u += 4)
                    *reinterpret_cast<float4*>(buf + B::V + tid * 8 + u) = make_float4(f[u], f[u + 1], f[u + 2], f[u + 3]);
            }
        } else {
#pragma unroll
            for (int e = 0; e < N8 * 8; ++e) {
                const int i = tid + e * SCAN_THREADS, t = i / DIMP, d = i - t * DIMP;
                if (t < CK) {
                    const int at = t * B::ROW + (d / RPT) * B::PART + d % RPT;
                    buf[B::Q + at] = to_f(sq[e]) * (iq[e] * q_scale);
                    buf[B::K + at] = to_f(sk[e]) * ik[e];
                }
            }
#pragma unroll
            for (int e = 0; e < CK * COLS / SCAN_THREADS; ++e) buf[B::V + tid + e * SCAN_THREADS] = to_f(sv[e]);
        }
        // T and A: rows of 16 into rows of MAT; then P and D
        const int i = tid * 4, r = i / CK;                    // 0 .. 511: T's rows, then A's
        *reinterpret_cast<float4*>(buf + B::T + r * MAT + (i & (CK - 1))) = rm[0];
        if (tid < RECORD / 4 - SCAN_THREADS) *reinterpret_cast<float4*>(buf + B::P + tid * 4) = rm[1];
    };
    fetch(0);
    put(sm);
    __syncthreads();
    int cur = 0;
    for (int t0 = 0; t0 < n; t0 += CK) {
        const int nt = min(CK, n - t0);
        const bool more = t0 + CK < n;
        const float* buf = sm + (AHEAD ? cur * B::FLOATS : 0);
        if (AHEAD && more) fetch(t0 + CK);
        // K S and Q S: TB rows at a time give eight sums per lane, value index = which * 4 + row * CPT + column
        constexpr int TB = 4 / CPT;
#pragma unroll 1
        for (int tt = 0; tt < CK; tt += TB) {
            float acc[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[i] = 0.f;
#pragma unroll
            for (int j = 0; j < RPT / 4; ++j)
#pragma unroll
                for (int r = 0; r < TB; ++r) {
                    const float4 k4 = *reinterpret_cast<const float4*>(buf + B::K + (tt + r) * B::ROW + part * B::PART + 4 * j);
                    const float4 q4 = *reinterpret_cast<const float4*>(buf + B::Q + (tt + r) * B::ROW + part * B::PART + 4 * j);
                    const float kv[4] = {k4.x, k4.y, k4.z, k4.w}, qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int u = 0; u < 4; ++u)
#pragma unroll
                        for (int c = 0; c < CPT; ++c) {
                            acc[r * CPT + c] += kv[u] * S[4 * j + u][c];
                            acc[4 + r * CPT + c] += qv[u] * S[4 * j + u][c];
                        }
                }
            // sums over the eight lanes: lane `part` ends with value `part`
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float mine = (part & 4) ? acc[4 + i] : acc[i], theirs = (part & 4) ? acc[i] : acc[4 + i];
                acc[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, 4);
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float mine = (part & 2) ? acc[2 + i] : acc[i], theirs = (part & 2) ? acc[i] : acc[2 + i];
                acc[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, 2);
            }
            const float mine = (part & 1) ? acc[1] : acc[0], theirs = (part & 1) ? acc[0] : acc[1];
            const float sum = mine + __shfl_xor_sync(0xffffffffu, theirs, 1);
            const int r = (part & 3) / CPT, c = (part & 3) % CPT, wc = (lane / SHARE) * CPT + c;
            (part & 4 ? wq : wk)[(tt + r) * B::WCOLS + wc] = sum;
        }
        __syncwarp();
        // per warp: X = V - P K S; U = T X; O = P Q S + A U.  A lane has two rows and CPT columns of WCOLS.
        const int r0 = (lane >> 2) * 2, wc = lane & 3;
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const int at = (r0 + r) * B::WCOLS + wc + 4 * c;
                wk[at] = buf[B::V + (r0 + r) * COLS + warp * B::WCOLS + wc + 4 * c] - buf[B::P + r0 + r] * wk[at];
            }
        __syncwarp();
        float u[2][CPT], o[2][CPT];
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                u[r][c] = 0.f;
                o[r][c] = buf[B::P + r0 + r] * wq[(r0 + r) * B::WCOLS + wc + 4 * c];
            }
#pragma unroll
        for (int j = 0; j < CK; j += 4) {
            const float4 m0 = *reinterpret_cast<const float4*>(buf + B::T + r0 * MAT + j);
            const float4 m1 = *reinterpret_cast<const float4*>(buf + B::T + (r0 + 1) * MAT + j);
            const float a0[4] = {m0.x, m0.y, m0.z, m0.w}, a1[4] = {m1.x, m1.y, m1.z, m1.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    const float x = wk[(j + i) * B::WCOLS + wc + 4 * c];
                    u[0][c] += a0[i] * x;
                    u[1][c] += a1[i] * x;
                }
        }
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int c = 0; c < CPT; ++c) wu[(r0 + r) * B::WCOLS + wc + 4 * c] = u[r][c];
        __syncwarp();
#pragma unroll
        for (int j = 0; j < CK; j += 4) {
            const float4 m0 = *reinterpret_cast<const float4*>(buf + B::A + r0 * MAT + j);
            const float4 m1 = *reinterpret_cast<const float4*>(buf + B::A + (r0 + 1) * MAT + j);
            const float a0[4] = {m0.x, m0.y, m0.z, m0.w}, a1[4] = {m1.x, m1.y, m1.z, m1.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    const float x = wu[(j + i) * B::WCOLS + wc + 4 * c];
                    o[0][c] += a0[i] * x;
                    o[1][c] += a1[i] * x;
                }
        }
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const int oc = c0 + warp * B::WCOLS + wc + 4 * c;
                if (r0 + r < nt && oc < vdim) out[(size_t)(row0 + t0 + r0 + r) * ldo + (size_t)h * vdim + oc] = o[r][c];
            }
        // the state: S = P_16 S + sum_t (D_16,t u_t) k_t
        const float pc = buf[B::P + CK - 1];
#pragma unroll
        for (int r = 0; r < RPT; ++r)
#pragma unroll
            for (int c = 0; c < CPT; ++c) S[r][c] *= pc;
#pragma unroll 4
        for (int t = 0; t < CK; ++t) {
            const float dt = buf[B::D + t];
            float uc[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) uc[c] = dt * wu[t * B::WCOLS + (lane / SHARE) * CPT + c];
#pragma unroll
            for (int j = 0; j < RPT / 4; ++j) {
                const float4 k4 = *reinterpret_cast<const float4*>(buf + B::K + t * B::ROW + part * B::PART + 4 * j);
                const float kv[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int e = 0; e < 4; ++e)
#pragma unroll
                    for (int c = 0; c < CPT; ++c) S[4 * j + e][c] += kv[e] * uc[c];
            }
        }
        __syncwarp();
        if (more) {
            if (AHEAD) {
                put(sm + (cur ^ 1) * B::FLOATS);              // nobody reads that buffer: its chunk was walked a round ago
                cur ^= 1;
            } else {
                __syncthreads();
                fetch(t0 + CK);
                put(sm);
            }
            __syncthreads();
        }
    }
#pragma unroll
    for (int r = 0; r < RPT; ++r)
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const int i = part * RPT + r;
            if (i < dim && col + c < vdim) my_state[(size_t)i * vdim + c] = S[r][c];
        }
}

constexpr size_t ALONE_BYTES = 120 * 1024;

int sm_count() {
    static int n = 0;
    if (n == 0) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) n = 148;
    }
    return n;
}

template <typename T, int RPT, int CPT, bool VEC>
int scan_as(const void* q, const void* k, const void* v, long long ld, const float* inv, int ldi, float q_scale, const float* rec,
            const int* seq_row0, const int* seq_len, const int* slots, float* state, long long slot_stride, float* out,
            long long ldo, int B, int H, int G, int dim, int vdim, cudaStream_t st) {
    using Buf = ScanBuf<RPT, CPT>;
    // A block walks its sequence alone, so the scan takes as long as the slowest block: two on one SM while others are idle (the
    // kernel in front still fills them when blocks are handed out) would set the pace.  Blocks that all fit one by one ask for
    // more than half of an SM's shared memory.
    const dim3 grid((vdim + Buf::COLS - 1) / Buf::COLS, H, B);
    const bool alone = (long long)grid.x * H * B <= sm_count();
    const size_t need = Buf::bytes(RPT <= 16 ? 2 : 1), smem = alone && need < ALONE_BYTES ? ALONE_BYTES : need;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(delta_scan_kernel<T, RPT, CPT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             (int)(need > ALONE_BYTES ? need : ALONE_BYTES));
        set = true;
    }
    launch_pdl(delta_scan_kernel<T, RPT, CPT, VEC>, grid, dim3(SCAN_THREADS), smem, st,
               (const T*)q, (const T*)k, (const T*)v, ld, inv, ldi, q_scale, rec, seq_row0, seq_len, slots, state, slot_stride, out,
               ldo, H, G, dim, vdim);
    QNN_LAUNCH_CHECK();
}

// ---- one token per sequence -------------------------------------------------------------------------------------
// A cluster of `splits` CTAs has one (sequence, value head); a CTA has `cw` of its value columns.  Everything is asked for
// before the wait for the kernel in front but what that kernel writes: the state (the largest part), the ring of the
// convolution's last inputs, filters, the gates' weights.  The CTAs of a cluster exchange their sums of squares for the
// output norm through distributed shared memory.
constexpr int STEP_THREADS = 256;

struct StepArgs {
    const void* p;              // rows of the input product: q | k | v | gate
    long long ldp;
    const void* x;              // [B, W]: the layer's normed input, for the gates' products
    const void* w_ba;           // [2 H, W]
    int W, w_dt;
    const void* conv;           // [C, taps]
    int c_dt, taps;
    const float* rate;          // exp(A)
    const float* bias;
    const void* norm;           // [vdim]
    int n_dt;
    float eps, q_scale, unit_eps;
    float* state;               // slot s: state + s * slot_stride: [taps][C]; from float s_off on [H][dim][vdim]
    long long slot_stride, s_off;
    const int* tok_pos;
    const int* slots;
    void* out;                  // [B, ldo]: H * vdim columns
    long long ldo;
    int B, H, G, dim, vdim, cw;
};

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ unsigned cluster_rank() {
    unsigned r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}

// VEC: the CTA's columns lie in fours on 16 bytes; RPT: state rows per thread
template <typename T, int RPT, bool VEC>
__global__ void __launch_bounds__(STEP_THREADS)
delta_step_kernel(const StepArgs a, int splits) {
    constexpr int V = VEC ? 4 : 1;
    constexpr int CG = 16;                                    // threads side by side over columns: CG * V columns at most
    constexpr int RG = STEP_THREADS / CG;                     // row groups
    __shared__ float sk[MAX_DIM], sq[MAX_DIM], sv[CG * V], su[CG * V];
    __shared__ float red[8][6];
    __shared__ float part[2][8][CG * V];
    __shared__ float squares[8];                              // by rank of the cluster
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = (int)(blockIdx.x % splits), h = (int)(blockIdx.x / splits), b = blockIdx.y;
    const int g = h / (a.H / a.G), D = a.dim, VD = a.vdim;
    const int c0 = split * a.cw, ncol = max(0, min(a.cw, VD - c0));
    const int C = 2 * a.G * D + a.H * VD;
    const int slot = a.slots[b], pos = a.tok_pos[b];
    const int cg = tid % CG, rg = tid / CG;
    if (splits > 1) cluster_arrive();                         // the other CTAs' shared memory is there (waited for below)
    const bool live = slot >= 0;
    float* base = a.state + (size_t)(live ? slot : 0) * a.slot_stride;
    float* S0 = base + a.s_off + (size_t)h * D * VD + c0;
    // the state: rows rg, rg + RG, ..; columns cg * V ..
    float S[RPT][V];
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rg + r * RG;
#pragma unroll
        for (int c = 0; c < V; ++c) S[r][c] = 0.f;
        if (live && i < D && cg * V < ncol) {
            if (VEC) {
                const float4 s4 = *reinterpret_cast<const float4*>(S0 + (size_t)i * VD + cg * 4);
                S[r][0] = s4.x; S[r][1 % V] = s4.y; S[r][2 % V] = s4.z; S[r][3 % V] = s4.w;
            } else {
                S[r][0] = S0[(size_t)i * VD + cg];
            }
        }
    }
    // channels of the convolution that this CTA needs: q of its head, k of its head, its value columns.  Two or three per thread
    // at most (dim <= 256); a channel's past inputs and its filter are summed up to the newest tap here.
    const int nch = 2 * D + ncol;
    constexpr int PER = (2 * MAX_DIM + CG * V + STEP_THREADS - 1) / STEP_THREADS;
    float past[PER], last[PER];
    int chan[PER];
#pragma unroll
    for (int e = 0; e < PER; ++e) {
        const int i = tid + e * STEP_THREADS;
        past[e] = last[e] = 0.f;
        chan[e] = -1;
        if (i < nch) {
            const int ch = i < D ? g * D + i : (i < 2 * D ? a.G * D + g * D + (i - D) : 2 * a.G * D + h * VD + c0 + (i - 2 * D));
            chan[e] = ch;
            last[e] = load_as_f(a.conv, a.c_dt, (size_t)ch * a.taps + a.taps - 1);
            if (live)
                for (int j = 0; j + 1 < a.taps; ++j) {
                    const int at = pos - a.taps + 1 + j;
                    if (at >= 0) past[e] = fmaf(load_as_f(a.conv, a.c_dt, (size_t)ch * a.taps + j), base[(size_t)(at % a.taps) * C + ch], past[e]);
                }
        }
    }
    const float rate = a.rate[h], bias = a.bias[h];
    pdl_wait();
    const T* prow = (const T*)a.p + (size_t)b * a.ldp;
    const T* xrow = (const T*)a.x + (size_t)b * a.W;
    float raw[PER];
#pragma unroll
    for (int e = 0; e < PER; ++e) raw[e] = chan[e] >= 0 ? to_f(prow[chan[e]]) : 0.f;
    // the gates' products
    float db = 0.f, da = 0.f;
    const size_t wb = (size_t)h * a.W, wa = (size_t)(a.H + h) * a.W;
    if (a.W % 8 == 0) {
        for (int i = tid * 8; i < a.W; i += STEP_THREADS * 8) {
            float xf[8], f[8], e8[8];
            load8_as_f(xrow, sizeof(T) == 2 ? QNN_DT_BF16 : QNN_DT_F32, i, xf);
            load8_as_f(a.w_ba, a.w_dt, wb + i, f);
            load8_as_f(a.w_ba, a.w_dt, wa + i, e8);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                db += xf[j] * f[j];
                da += xf[j] * e8[j];
            }
        }
    } else {
        for (int i = tid; i < a.W; i += STEP_THREADS) {
            const float xf = to_f(xrow[i]);
            db += xf * load_as_f(a.w_ba, a.w_dt, wb + i);
            da += xf * load_as_f(a.w_ba, a.w_dt, wa + i);
        }
    }
    // convolution, silu (rounded as a prompt's rows are stored), the ring's newest row
    float ssq = 0.f, ssk = 0.f;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
        const int i = tid + e * STEP_THREADS;
        if (chan[e] >= 0) {
            const float y = to_f(from_f<T>(silu(fmaf(last[e], raw[e], past[e]))));
            if (i < D) { sq[i] = y; ssq += y * y; }
            else if (i < 2 * D) { sk[i - D] = y; ssk += y * y; }
            else sv[i - 2 * D] = y;
            // q and k belong to all heads of the group and all CTAs of a cluster: one of them keeps them
            const bool keeper = i >= 2 * D || (split == 0 && h % (a.H / a.G) == 0);
            if (live && keeper) base[(size_t)(pos % a.taps) * C + chan[e]] = raw[e];
        }
    }
    {
        const float s0 = warp_sum(ssq), s1 = warp_sum(ssk), s2 = warp_sum(db), s3 = warp_sum(da);
        if (lane == 0) { red[warp][0] = s0; red[warp][1] = s1; red[warp][2] = s2; red[warp][3] = s3; }
    }
    __syncthreads();
    float tq = 0.f, tk = 0.f, tb = 0.f, ta = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) { tq += red[w][0]; tk += red[w][1]; tb += red[w][2]; ta += red[w][3]; }
    const float fq = rsqrtf(tq + a.unit_eps) * a.q_scale, fk = rsqrtf(tk + a.unit_eps);
    const float beta = beta_of(tb), gate = decay_of(ta, rate, bias);
    // S^T k and S^T q: partial sums over a thread's rows, the two row groups of a warp by shuffle, the warps through shared memory
    float mk[V], mq[V], kr[RPT], kq = 0.f;
#pragma unroll
    for (int c = 0; c < V; ++c) mk[c] = mq[c] = 0.f;
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rg + r * RG;
        const float k1 = i < D ? sk[i] * fk : 0.f, q1 = i < D ? sq[i] * fq : 0.f;
        kr[r] = k1;
        if (cg == 0) kq += k1 * q1;
#pragma unroll
        for (int c = 0; c < V; ++c) {
            mk[c] += k1 * S[r][c];
            mq[c] += q1 * S[r][c];
        }
    }
#pragma unroll
    for (int c = 0; c < V; ++c) {
        mk[c] += __shfl_xor_sync(0xffffffffu, mk[c], 16);
        mq[c] += __shfl_xor_sync(0xffffffffu, mq[c], 16);
        if (lane < CG) {
            part[0][warp][cg * V + c] = mk[c];
            part[1][warp][cg * V + c] = mq[c];
        }
    }
    kq += __shfl_xor_sync(0xffffffffu, kq, 16);
    if (lane == 0) red[warp][4] = kq;
    __syncthreads();
    float o = 0.f;
    if (tid < CG * V) {
        float s0 = 0.f, s1 = 0.f, s2 = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) { s0 += part[0][w][tid]; s1 += part[1][w][tid]; s2 += red[w][4]; }
        const float u = tid < ncol ? beta * (sv[tid] - gate * s0) : 0.f;
        su[tid] = u;
        o = tid < ncol ? gate * s1 + s2 * u : 0.f;
    }
    float oo = o * o;                                         // threads of the first CG * V only: at most two warps
    oo = warp_sum(oo);
    if (lane == 0) red[warp][5] = oo;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) total += red[w][5];
    if (splits > 1) {
        cluster_wait();
        if (tid < splits) {                                   // this CTA's sum to every rank
            unsigned local = (unsigned)__cvta_generic_to_shared(&squares[cluster_rank()]), remote;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"((unsigned)tid));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(total) : "memory");
        }
        cluster_arrive();
    }
    // meanwhile the new state
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rg + r * RG;
        if (live && i < D && cg * V < ncol) {
            if (VEC) {
                float4 s4;
                s4.x = gate * S[r][0] + kr[r] * su[cg * V];
                s4.y = gate * S[r][1 % V] + kr[r] * su[cg * V + 1 % V];
                s4.z = gate * S[r][2 % V] + kr[r] * su[cg * V + 2 % V];
                s4.w = gate * S[r][3 % V] + kr[r] * su[cg * V + 3 % V];
                *reinterpret_cast<float4*>(S0 + (size_t)i * VD + cg * 4) = s4;
            } else {
                S0[(size_t)i * VD + cg] = gate * S[r][0] + kr[r] * su[cg];
            }
        }
    }
    if (splits > 1) {
        cluster_wait();
        total = 0.f;
        for (int r = 0; r < splits; ++r) total += squares[r];
    }
    if (tid < ncol) {
        const float y = o * rsqrtf(total / (float)VD + a.eps) * load_as_f(a.norm, a.n_dt, c0 + tid);
        const float z = to_f(prow[C + h * VD + c0 + tid]);
        ((T*)a.out)[(size_t)b * a.ldo + (size_t)h * VD + c0 + tid] = from_f<T>(live ? y * silu(z) : 0.f);
    }
}

template <typename T, int RPT, bool VEC>
int step_as(const StepArgs& a, int splits, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)(a.H * splits), (unsigned)a.B);
    cfg.blockDim = dim3(STEP_THREADS);
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (splits > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = (unsigned)splits;
        attr[n].val.clusterDim.y = 1;
        attr[n].val.clusterDim.z = 1;
        ++n;
    }
    if (pdl_enabled() && (long long)a.H * splits * a.B <= pdl_max_grid()) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    const cudaError_t rc = cudaLaunchKernelEx(&cfg, delta_step_kernel<T, RPT, VEC>, a, splits);
    if (rc != cudaSuccess) return (int)rc;
    QNN_LAUNCH_CHECK();
}

template <typename T, bool VEC>
int step_rows(const StepArgs& a, int splits, cudaStream_t st) {
    const int rpt = (a.dim + 15) / 16;
    if (rpt <= 4) return step_as<T, 4, VEC>(a, splits, st);
    if (rpt <= 8) return step_as<T, 8, VEC>(a, splits, st);
    return step_as<T, 16, VEC>(a, splits, st);
}

}  // namespace

// q, k: [rows, G * dim], v: [rows, H * vdim] of `dtype`, one row pitch `ld`; inv: [rows, ldi] with 1 / length of the G query heads,
// then of the G key heads; seq_row0, seq_len: first row and row count of the B sequences (both null: row b alone); pre: [rows, ldp] with b of the H heads, then a of the H heads; rate, bias: [H] float32 (rate =
// exp(A)); rec: at least (T / 16 + B) * H records of 544 floats.  longest: the most rows of a sequence.  dim up to 256.
QNN_API int qnn_delta_chunks(const void* q, const void* k, long long ld, int dtype, const float* inv, int ldi, const float* pre,
                             int ldp, const float* rate, const float* bias, float q_scale, const int* seq_row0, const int* seq_len,
                             float* rec, int B, int longest, int H, int G, int dim, cudaStream_t st) {
    if (B <= 0 || longest <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || dim <= 0 || dim > MAX_DIM || B > 65535 || G > 65535 || ldi < 2 * G || ldp < 2 * H)
        return QNN_ERR_ARGUMENT;
    if ((seq_row0 == nullptr) != (seq_len == nullptr)) return QNN_ERR_ARGUMENT;
    const int pitch = ((dim + 3) & ~3) + 4;
    const size_t smem = ((size_t)2 * CK * pitch + 6 * CK * (CK + 1)) * sizeof(float);
    if (smem > 48 * 1024) return QNN_ERR_UNSUPPORTED;
    const dim3 grid((unsigned)((longest + CK - 1) / CK), G, B);
    if (dtype == QNN_DT_BF16)
        launch_pdl(delta_chunks_kernel<bf16>, grid, dim3(128), smem, st, (const bf16*)q, (const bf16*)k, ld, inv, ldi, pre, ldp,
                   rate, bias, q_scale, seq_row0, seq_len, rec, H, G, dim);
    else
        launch_pdl(delta_chunks_kernel<float>, grid, dim3(128), smem, st, (const float*)q, (const float*)k, ld, inv, ldi, pre, ldp,
                   rate, bias, q_scale, seq_row0, seq_len, rec, H, G, dim);
    QNN_LAUNCH_CHECK();
}

// The same rows; slots: the state slot of each sequence (negative: nothing is read or written); state: slot s's
// [H, dim, vdim] floats at state + s * slot_stride; out: [rows, ldo] float32, H * vdim columns; cpt: 16 or 32 value columns per
// block (1 or 2: many sequences fill the device with the wider ones, which read the rows half as often).
QNN_API int qnn_delta_scan(const void* q, const void* k, const void* v, long long ld, int dtype, const float* inv, int ldi,
                           float q_scale, const float* rec, const int* seq_row0, const int* seq_len, const int* slots, float* state,
                           long long slot_stride, float* out, long long ldo, int B, int H, int G, int dim, int vdim, int cpt,
                           cudaStream_t st) {
    if (B <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || dim <= 0 || dim > MAX_DIM || vdim <= 0 || B > 65535 || H > 65535 || ldi < 2 * G ||
        slot_stride < (long long)H * dim * vdim || (cpt != 1 && cpt != 2) || (seq_row0 == nullptr) != (seq_len == nullptr))
        return QNN_ERR_ARGUMENT;
    const size_t es = dtype == QNN_DT_BF16 ? 2 : 4;
    const bool vec = dim % 8 == 0 && vdim % 8 == 0 && (ld * es) % 16 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15) == 0;
    const int rpt = (dim + SHARE - 1) / SHARE;
#define QNN_DS(T, R, C, VV) \
    return scan_as<T, R, C, VV>(q, k, v, ld, inv, ldi, q_scale, rec, seq_row0, seq_len, slots, state, slot_stride, out, ldo, B, H, \
                                G, dim, vdim, st)
#define QNN_DS_COLS(T, R, VV)        \
    if (cpt == 2) QNN_DS(T, R, 2, VV); \
    else QNN_DS(T, R, 1, VV);
#define QNN_DS_ROWS(T, VV)                        \
    if (rpt <= 4) { QNN_DS_COLS(T, 4, VV) }       \
    else if (rpt <= 8) { QNN_DS_COLS(T, 8, VV) }  \
    else if (rpt <= 16) { QNN_DS_COLS(T, 16, VV) } \
    else { QNN_DS_COLS(T, 32, VV) }
    if (dtype == QNN_DT_BF16) {
        if (vec) { QNN_DS_ROWS(bf16, true) } else { QNN_DS_ROWS(bf16, false) }
    } else {
        if (vec) { QNN_DS_ROWS(float, true) } else { QNN_DS_ROWS(float, false) }
    }
#undef QNN_DS_ROWS
#undef QNN_DS_COLS
#undef QNN_DS
}

// p: [B, ldp] rows q | k | v | gate of the input product; x: [B, W] the product's input; w_ba: [2 H, W]; conv: [2 G dim + H vdim,
// taps]; state: slot s at state + s * slot_stride: [taps][channels] the ring of last inputs (position p in row p mod taps), from
// float s_off on [H][dim][vdim]; slots negative: a row of no sequence (its output is zero).  out: [B, ldo] of `dtype`.
QNN_API int qnn_delta_step(const void* p, int dtype, long long ldp, const void* x, int W, const void* w_ba, int w_dt,
                           const void* conv, int c_dt, int taps, const float* rate, const float* bias, const void* norm, int n_dt,
                           float eps, float unit_eps, float q_scale, float* state, long long slot_stride, long long s_off, const int* tok_pos,
                           const int* slots, void* out, long long ldo, int B, int H, int G, int dim, int vdim, cudaStream_t st) {
    if (B <= 0) return 0;
    const long long C = 2LL * G * dim + (long long)H * vdim;
    if (H <= 0 || G <= 0 || H % G || dim <= 0 || vdim <= 0 || taps < 1 || W <= 0 || ldp < C + (long long)H * vdim ||
        s_off < taps * C || slot_stride < s_off + (long long)H * dim * vdim || B > 65535 || ldo < (long long)H * vdim)
        return QNN_ERR_ARGUMENT;
    if (dim > MAX_DIM) return QNN_ERR_UNSUPPORTED;
    if (W % 8 == 0 && (((uintptr_t)x | (uintptr_t)w_ba) & 15)) return QNN_ERR_ARGUMENT;
    // columns of a CTA: up to 64 in fours, up to 16 one by one; at most eight CTAs share a head
    const bool vec = vdim % 4 == 0 && s_off % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    const int most = vec ? 64 : 16;
    int splits = 1;
    while (splits < 8 && (long long)splits * most < vdim) splits *= 2;
    int cw = (vdim + splits - 1) / splits;
    if (vec) cw = (cw + 3) / 4 * 4;
    if (cw > most) return QNN_ERR_UNSUPPORTED;
    StepArgs a = {p, ldp, x, w_ba, W, w_dt, conv, c_dt, taps, rate, bias, norm, n_dt, eps, q_scale, unit_eps, state, slot_stride, s_off,
                  tok_pos, slots, out, ldo, B, H, G, dim, vdim, cw};
    if (dtype == QNN_DT_BF16) return vec ? step_rows<bf16, true>(a, splits, st) : step_rows<bf16, false>(a, splits, st);
    return vec ? step_rows<float, true>(a, splits, st) : step_rows<float, false>(a, splits, st);
}
