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
//   qnn_delta_scan     walks the chunks of every sequence in order, from the slot's state and back into it; bfloat16 rows on the
//                      tensor cores with every float32 matrix in three bfloat16 parts, others on the FMA pipes
// (One token per sequence: delta_step.cu.)
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
#include "delta_rule.cuh"

using namespace qnn;

namespace {

constexpr int CK = 16;                       // rows of a chunk
constexpr int RECORD = 2 * CK * CK + 2 * CK; // floats that qnn_delta_chunks leaves per (chunk, value head): T, A, P, D

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

// ---- bfloat16 rows: the same on the tensor cores ---------------------------------------------------------------------
// Keys and queries are bfloat16 numbers times a float32 factor per row, so a float32 matrix meets them on the tensor cores
// without loss when it is cut into three bfloat16 numbers per element (8 bits of its 24 each) and the factors are applied
// to the results: x = hi + mid + lo costs three products with one exact factor and six with another float32 matrix (the three
// smallest of nine terms lie below float32's rounding).  Accumulation is float32.
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// d = a b without an accumulator to start from
__device__ __forceinline__ void mma_first(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%10,%10,%10,%10};\n"
        : "=f"(d[0]), "=f"(d[1]), "=f"(d[2]), "=f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1), "f"(0.f));
}
__device__ __forceinline__ float low_of(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float high_of(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
struct Split3 { uint32_t h[4], m[4], l[4]; };
// The upper half of a float32 is a bfloat16 with its first 8 significant bits; what is left has 16, and once more 8: the three
// parts add up to the number exactly (but for what lies below float32's smallest normal numbers).
__device__ __forceinline__ float upper(float x) { return __uint_as_float(__float_as_uint(x) & 0xffff0000u); }
__device__ __forceinline__ uint32_t uppers(float a, float b) { return __byte_perm(__float_as_uint(a), __float_as_uint(b), 0x7632); }
__device__ __forceinline__ void split(float a, float b, uint32_t& h, uint32_t& m, uint32_t& l) {
    h = uppers(a, b);
    a -= upper(a);
    b -= upper(b);
    m = uppers(a, b);
    l = uppers(a - upper(a), b - upper(b));
}
// two accumulator tiles (16 x 8 each, side by side) as the A operand of a product over those 16 columns
__device__ __forceinline__ void split_tiles(const float (&x)[4], const float (&y)[4], Split3& s) {
    split(x[0], x[1], s.h[0], s.m[0], s.l[0]);
    split(x[2], x[3], s.h[1], s.m[1], s.l[1]);
    split(y[0], y[1], s.h[2], s.m[2], s.l[2]);
    split(y[2], y[3], s.h[3], s.m[3], s.l[3]);
}
__device__ __forceinline__ void cp16(unsigned dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src) : "memory");
}

// What a chunk leaves for the scan, per value head: T and A in three bfloat16 matrices each ([3][2][16][8]: row t of the columns
// j = 8 c .. 8 c + 7, c = 0, 1, so that the eight rows of an ldmatrix lie side by side), then per row P_t / |k_t|,
// P_t q_scale / |q_t|, D_16,t / |k_t|, and P_16: 3280 bytes.
constexpr int TC_T = 0, TC_A = 3 * CK * CK * 2, TC_F = 2 * TC_A, TC_RECORD = TC_F + (3 * CK + 4) * 4;

// a warp per (chunk, query/key head)
__global__ void __launch_bounds__(128)
delta_chunks_tc_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k, long long ld, const float* __restrict__ inv, int ldi,
                       const float* __restrict__ pre, int ldp, const float* __restrict__ rate, const float* __restrict__ bias,
                       float q_scale, const int* __restrict__ seq_row0, const int* __restrict__ seq_len,
                       unsigned char* __restrict__ rec, int H, int G, int dim) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, j = lane & (CK - 1), half = lane >> 4;
    const int dpad = (dim + 15) & ~15, pitch = dpad * 2 + 16;
    const int own = 2 * CK * pitch + 3 * CK * (CK + 1) * 4;
    unsigned char* mine = smem + (size_t)warp * own;
    float* kk = reinterpret_cast<float*>(mine + 2 * CK * pitch);
    float* qk = kk + CK * (CK + 1);
    float* L = qk + CK * (CK + 1);
    const int c = blockIdx.x * 4 + warp, g = blockIdx.y, b = blockIdx.z;
    pdl_wait();
    const int n = seq_len != nullptr ? seq_len[b] : 1, row0 = seq_row0 != nullptr ? seq_row0[b] : b, t0 = c * CK;
    if (t0 >= n) return;                                      // (nothing below waits for another warp)
    const int nt = min(CK, n - t0);
    const int pieces = dpad / 8;
    const unsigned kb = (unsigned)__cvta_generic_to_shared(mine), qb = kb + CK * pitch;
    for (int i = lane; i < CK * pieces; i += 32) {
        const int t = i / pieces, d = (i - t * pieces) * 8;
        if (t < nt && d < dim) {
            const size_t at = (size_t)(row0 + t0 + t) * ld + (size_t)g * dim + d;
            cp16(kb + t * pitch + d * 2, k + at);
            cp16(qb + t * pitch + d * 2, q + at);
        } else {
            *reinterpret_cast<uint4*>(mine + t * pitch + d * 2) = make_uint4(0, 0, 0, 0);
            *reinterpret_cast<uint4*>(mine + (CK + t) * pitch + d * 2) = make_uint4(0, 0, 0, 0);
        }
    }
    float iq = 0.f, ik = 0.f;                                 // of row j
    if (j < nt) {
        const size_t row = (size_t)(row0 + t0 + j);
        iq = inv[row * ldi + g] * q_scale;
        ik = inv[row * ldi + G + g];
    }
    const int per = H / G;
    float zb = 0.f, za = 0.f;                                 // the first value head's logits, asked for with the rows
    if (j < nt) {
        const float* pr = pre + (size_t)(row0 + t0 + j) * ldp;
        zb = pr[g * per];
        za = pr[H + g * per];
    }
    asm volatile("cp.async.wait_all;\n" ::: "memory");
    __syncwarp();
    const int mi = lane >> 3, mr = lane & 7;                  // matrix and row that this lane addresses for ldmatrix
    float akk[2][4], aqk[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) akk[i][e] = aqk[i][e] = 0.f;
    for (int d = 0; d < dpad; d += 16) {
        uint32_t ka[4], qa[4], kn[4];
        ldsm4(ka, kb + ((mi & 1) * 8 + mr) * pitch + (d + (mi >> 1) * 8) * 2);      // rows as A
        ldsm4(qa, qb + ((mi & 1) * 8 + mr) * pitch + (d + (mi >> 1) * 8) * 2);
        ldsm4(kn, kb + ((mi >> 1) * 8 + mr) * pitch + (d + (mi & 1) * 8) * 2);      // rows as B
        mma(akk[0], ka, kn[0], kn[1]);
        mma(akk[1], ka, kn[2], kn[3]);
        mma(aqk[0], qa, kn[0], kn[1]);
        mma(aqk[1], qa, kn[2], kn[3]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int t = (lane >> 2) + (e >> 1) * 8, col = i * 8 + (lane & 3) * 2 + (e & 1);
            const float kt = __shfl_sync(0xffffffffu, ik, t), qt = __shfl_sync(0xffffffffu, iq, t), kj = __shfl_sync(0xffffffffu, ik, col);
            kk[t * (CK + 1) + col] = akk[i][e] * (kt * kj);
            qk[t * (CK + 1) + col] = aqk[i][e] * (qt * kj);
        }
    __syncwarp();
    for (int s = 0; s < per; ++s) {
        const int h = g * per + s;
        unsigned char* out = rec + (record_of(row0, b, c) * H + h) * TC_RECORD;
        bf16* oT = reinterpret_cast<bf16*>(out + TC_T);
        bf16* oA = reinterpret_cast<bf16*>(out + TC_A);
        float* oF = reinterpret_cast<float*>(out + TC_F);
        float be = 0.f, ga = 1.f;
        if (j < nt) {
            be = beta_of(zb);
            ga = decay_of(za, rate[h], bias[h]);
            if (s + 1 < per) {
                const float* pr = pre + (size_t)(row0 + t0 + j) * ldp;
                zb = pr[h + 1];
                za = pr[H + h + 1];
            }
        }
        auto put = [&](bf16* m, int t, float v) {
            const float r = v - upper(v), s = r - upper(r);
            const int at = (j >> 3) * (CK * 8) + t * 8 + (j & 7);
            m[at] = __ushort_as_bfloat16((unsigned short)(__float_as_uint(v) >> 16));
            m[CK * CK + at] = __ushort_as_bfloat16((unsigned short)(__float_as_uint(r) >> 16));
            m[2 * CK * CK + at] = __ushort_as_bfloat16((unsigned short)(__float_as_uint(s) >> 16));
        };
        float d = 1.f, p = 1.f, mine_p = 1.f;
#pragma unroll
        for (int t = 0; t < CK; ++t) {
            const float gt = __shfl_sync(0xffffffffu, ga, t), bt = __shfl_sync(0xffffffffu, be, t);
            if (t > j) d *= gt;
            p *= gt;
            if (t == j) mine_p = p;
            if (half == 0) L[t * (CK + 1) + j] = t > j ? bt * d * kk[t * (CK + 1) + j] : 0.f;
            else put(oA, t, t >= j ? d * qk[t * (CK + 1) + j] : 0.f);
        }
        if (half == 0) {
            oF[j] = mine_p * ik;
            oF[CK + j] = mine_p * iq;
            oF[2 * CK + j] = d * ik;
            if (j < 4) oF[3 * CK + j] = p;
        }
        __syncwarp();
        if (half == 0) {
            float x[CK];
#pragma unroll
            for (int t = 0; t < CK; ++t) {
                float s0 = t == j ? 1.f : 0.f;
#pragma unroll
                for (int i = 0; i < t; ++i) s0 -= L[t * (CK + 1) + i] * x[i];
                x[t] = s0;
                put(oT, t, s0 * be);
            }
        }
        __syncwarp();
    }
}

// The scan.  A block owns 16 value columns of one (sequence, head) as S^T, 16 columns x key channels.  Four warps have a quarter
// of the key channels each (KS times 16) as accumulator tiles, which serve as the A operand of the products with keys and queries
// when they are split; their partial K S meet in shared memory (one barrier per chunk), and each of the four then forms X, U = T X
// and its quarter of the update by itself, all in registers.  Q S is formed in the shadow of that; two more warps take alternate
// chunks and turn it into the outputs a chunk later; the last two fetch chunks ahead, keys and values the one, queries and what
// qnn_delta_chunks left the other.
constexpr int TC_WORKERS = 4, TC_READERS = 2, TC_LOADERS = 2;
constexpr int TC_THREADS = 32 * (TC_WORKERS + TC_READERS + TC_LOADERS), TC_STAGES = 6, TC_AHEAD = TC_STAGES - 2;

template <bool V> struct Flag { static constexpr bool value = V; };

template <int KS>
struct TcStage {
    static constexpr int PITCH = KS * 128 + 16, VPITCH = 48;   // bytes: rows four banks apart
    static constexpr int K = 0, Q = CK * PITCH, V = 2 * CK * PITCH, R = V + CK * VPITCH, BYTES = R + TC_RECORD;
    static constexpr int RED = TC_STAGES * BYTES;              // [2][k, q][workers][2 tiles][32 lanes] float4
    static constexpr int TOTAL = RED + 2 * 2 * TC_WORKERS * 2 * 32 * 16;
    static_assert(BYTES % 16 == 0, "stages on 16 bytes");
};

template <int KS>
__global__ void __launch_bounds__(TC_THREADS, KS <= 2 ? 2 : 1)
delta_scan_tc_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k, const bf16* __restrict__ v, long long ld,
                     const unsigned char* __restrict__ rec, const int* __restrict__ seq_row0, const int* __restrict__ seq_len,
                     const int* __restrict__ slots, float* __restrict__ state, long long slot_stride, float* __restrict__ out,
                     long long ldo, int H, int G, int dim, int vdim) {
    using St = TcStage<KS>;
    extern __shared__ __align__(16) unsigned char smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, t4 = lane & 3, gr = lane >> 2, mi = lane >> 3, mr = lane & 7;
    const int h = blockIdx.y, c0 = blockIdx.x * 16, b = blockIdx.z;
    for (int i = tid; i < St::RED / 16; i += TC_THREADS) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
    pdl_wait();
    const int n = seq_len != nullptr ? seq_len[b] : 1, row0 = seq_row0 != nullptr ? seq_row0[b] : b, slot = slots[b];
    if (n <= 0) return;
    if (slot < 0) {                                           // rows of no sequence
        const int live = min(16, vdim - c0);
        for (int i = tid; i < n * live; i += TC_THREADS)
            out[(size_t)(row0 + i / live) * ldo + (size_t)h * vdim + c0 + i % live] = 0.f;
        return;
    }
    const int chunks = (n + CK - 1) / CK, g = h / (H / G);
    const unsigned base = (unsigned)__cvta_generic_to_shared(smem);
    float4* red = reinterpret_cast<float4*>(smem + St::RED);
    auto red_at = [&](int parity, int which, int w, int tile) { return red + (((parity * 2 + which) * TC_WORKERS + w) * 2 + tile) * 32 + lane; };
    __syncthreads();                                          // the stages are zero: rows and columns that nothing fills stay so
    if (warp >= TC_WORKERS + TC_READERS) {
        // ---- a loader.  Rows beyond the sequence keep what an earlier chunk left (or zeros): finite numbers whose factors are 0
        const int pieces = dim / 8, vp = min(2, (vdim - c0) / 8);
        const bool first_half = warp == TC_WORKERS + TC_READERS;
        const bf16* rows = first_half ? k : q;
        const int into = first_half ? St::K : St::Q;
        const int at_once = 32 / pieces, tl = lane / pieces, dl = lane - tl * pieces;        // rows side by side; this lane's
        auto load = [&](int c) {
            if (c < chunks) {
                const unsigned st = base + (c % TC_STAGES) * St::BYTES;
                const int nt = min(CK, n - c * CK);
                const size_t first = (size_t)(row0 + c * CK);
                if (tl < at_once) {
                    size_t at = (first + tl) * ld + (size_t)g * dim + dl * 8;
                    unsigned to = st + into + tl * St::PITCH + dl * 16;
                    for (int t = tl; t < nt; t += at_once, at += at_once * ld, to += at_once * St::PITCH) cp16(to, rows + at);
                }
                if (first_half) {
                    const int t = lane >> 1, p = lane & 1;
                    if (t < nt && p < vp)
                        cp16(st + St::V + t * St::VPITCH + p * 16, v + (first + t) * ld + (size_t)h * vdim + c0 + p * 8);
                } else {
                    const unsigned char* r = rec + (record_of(row0, b, c) * H + h) * TC_RECORD;
                    for (int i = lane; i < TC_RECORD / 16; i += 32) cp16(st + St::R + i * 16, r + i * 16);
                }
            }
            asm volatile("cp.async.commit_group;\n" ::: "memory");
        };
        for (int c = 0; c < TC_AHEAD; ++c) load(c);
        asm volatile("cp.async.wait_group %0;\n" ::"n"(TC_AHEAD - 1) : "memory");
        __syncthreads();
        for (int c = 0; c < chunks; ++c) {
            load(c + TC_AHEAD);                               // (the stage of chunk c - 2: everybody is past its barrier c - 1)
            asm volatile("cp.async.wait_group %0;\n" ::"n"(TC_AHEAD - 1) : "memory");
            __syncthreads();
        }
        __syncthreads();
        return;
    }
    // X^T = V^T - (P K S)^T of chunk c from the workers' partial sums, split for a product over the chunk's rows: first the
    // loads, then the rest, so that other work finds its place in between
    struct Parts { float4 m[2][TC_WORKERS]; float2 pk[2]; uint32_t v[4]; };
    auto fetch_x = [&](int c, Parts& p) {
        const unsigned st = base + (c % TC_STAGES) * St::BYTES;
        const float* f = reinterpret_cast<const float*>(smem + (c % TC_STAGES) * St::BYTES + St::R + TC_F);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int w = 0; w < TC_WORKERS; ++w) p.m[i][w] = *red_at(c & 1, 0, w, i);
#pragma unroll
        for (int i = 0; i < 2; ++i) p.pk[i] = *reinterpret_cast<const float2*>(f + i * 8 + t4 * 2);
        ldsm4t(p.v, st + St::V + ((mi >> 1) * 8 + mr) * St::VPITCH + (mi & 1) * 16);
    };
    auto form_x = [&](const Parts& p, Split3& x) {
        float xs[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float4 m = p.m[i][0];
#pragma unroll
            for (int w = 1; w < TC_WORKERS; ++w) {
                m.x += p.m[i][w].x; m.y += p.m[i][w].y; m.z += p.m[i][w].z; m.w += p.m[i][w].w;
            }
            xs[i][0] = low_of(p.v[2 * i]) - p.pk[i].x * m.x;
            xs[i][1] = high_of(p.v[2 * i]) - p.pk[i].y * m.y;
            xs[i][2] = low_of(p.v[2 * i + 1]) - p.pk[i].x * m.z;
            xs[i][3] = high_of(p.v[2 * i + 1]) - p.pk[i].y * m.w;
        }
        split_tiles(xs[0], xs[1], x);
    };
    // y += (x times the 16 x 16 matrix whose three parts are at `m`)^T, the small terms first
    auto times = [&](const Split3& x, const uint32_t (&mh)[4], const uint32_t (&mm)[4], const uint32_t (&ml)[4], float (&y)[2][4],
                     auto fresh) {                            // fresh: y starts from zero
        float z[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) mma_first(z[i], x.l, mh[2 * i], mh[2 * i + 1]);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            if constexpr (decltype(fresh)::value) mma_first(y[i], x.m, mh[2 * i], mh[2 * i + 1]);
            else mma(y[i], x.m, mh[2 * i], mh[2 * i + 1]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) mma(z[i], x.h, ml[2 * i], ml[2 * i + 1]);
#pragma unroll
        for (int i = 0; i < 2; ++i) mma(y[i], x.h, mm[2 * i], mm[2 * i + 1]);
#pragma unroll
        for (int i = 0; i < 2; ++i) mma(z[i], x.m, mm[2 * i], mm[2 * i + 1]);
#pragma unroll
        for (int i = 0; i < 2; ++i) mma(y[i], x.h, mh[2 * i], mh[2 * i + 1]);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[i][e] += z[i][e];
    };
    auto load_matrix = [&](int c, int at, uint32_t (&mh)[4], uint32_t (&mm)[4], uint32_t (&ml)[4]) {
        const unsigned a = base + (c % TC_STAGES) * St::BYTES + St::R + at + (mi & 1) * (CK * 16) + ((mi >> 1) * 8 + mr) * 16;
        ldsm4(mh, a);
        ldsm4(mm, a + CK * CK * 2);
        ldsm4(ml, a + 2 * CK * CK * 2);
    };
    if (warp >= TC_WORKERS) {
        // ---- the outputs: O = P Q S + A U, a chunk behind
        Split3 us;
        uint32_t ah[4], am[4], al[4];
        float2 pq[2];
        auto finish = [&](int c) {
            float o[2][4];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                float4 m = *red_at(c & 1, 1, 0, i);
#pragma unroll
                for (int w = 1; w < TC_WORKERS; ++w) {
                    const float4 x = *red_at(c & 1, 1, w, i);
                    m.x += x.x; m.y += x.y; m.z += x.z; m.w += x.w;
                }
                o[i][0] = pq[i].x * m.x;
                o[i][1] = pq[i].y * m.y;
                o[i][2] = pq[i].x * m.z;
                o[i][3] = pq[i].y * m.w;
            }
            times(us, ah, am, al, o, Flag<false>());
            const int nt = min(CK, n - c * CK);
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = i * 8 + t4 * 2 + (e & 1), col = c0 + gr + (e >> 1) * 8;
                    if (t < nt && col < vdim) out[(size_t)(row0 + c * CK + t) * ldo + (size_t)h * vdim + col] = o[i][e];
                }
        };
        __syncthreads();
        for (int c = 0; c < chunks; ++c) {
            __syncthreads();
            if ((c & 1) != warp - TC_WORKERS) {               // the other reader forms U of this chunk
                if (c > 0) finish(c - 1);
                continue;
            }
            Split3 x;
            {
                Parts p;
                fetch_x(c, p);
                form_x(p, x);
            }
            uint32_t th[4], tm[4], tl[4];
            load_matrix(c, TC_T, th, tm, tl);
            float u[2][4];
            times(x, th, tm, tl, u, Flag<true>());
            split_tiles(u[0], u[1], us);
            load_matrix(c, TC_A, ah, am, al);                 // (the stage may be filled anew before the outputs are formed)
            const float* f = reinterpret_cast<const float*>(smem + (c % TC_STAGES) * St::BYTES + St::R + TC_F);
#pragma unroll
            for (int i = 0; i < 2; ++i) pq[i] = *reinterpret_cast<const float2*>(f + CK + i * 8 + t4 * 2);
        }
        __syncthreads();
        if (((chunks - 1) & 1) == warp - TC_WORKERS) finish(chunks - 1);
        return;
    }
    // ---- a worker: key channels d0 .. d0 + 16 KS of S^T
    const int d0 = warp * KS * 16;
    float* my_state = state + (size_t)slot * slot_stride + (size_t)h * dim * vdim + c0;
    float S[2 * KS][4];
#pragma unroll
    for (int i = 0; i < 2 * KS; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = d0 + i * 8 + t4 * 2 + (e & 1), col = gr + (e >> 1) * 8;
            S[i][e] = (d < dim && c0 + col < vdim) ? my_state[(size_t)d * vdim + col] : 0.f;
        }
    __syncthreads();
    for (int c = 0; c < chunks; ++c) {
        const unsigned st = base + (c % TC_STAGES) * St::BYTES;
        const float* f = reinterpret_cast<const float*>(smem + (c % TC_STAGES) * St::BYTES + St::R + TC_F);
        Split3 s[KS];
        // S^T times the chunk's rows, over this warp's channels; the small parts have an accumulator of their own, which also
        // keeps products from waiting for one another
        auto product = [&](unsigned rows, float (&m)[2][4]) {
            float low[2][4];
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {
                uint32_t r[4];
                ldsm4(r, rows + ((mi >> 1) * 8 + mr) * St::PITCH + (d0 + ks * 16 + (mi & 1) * 8) * 2);
                if (ks == 0) {
                    mma_first(low[0], s[ks].l, r[0], r[1]);
                    mma_first(low[1], s[ks].l, r[2], r[3]);
                    mma_first(m[0], s[ks].h, r[0], r[1]);
                    mma_first(m[1], s[ks].h, r[2], r[3]);
                } else {
                    mma(low[0], s[ks].l, r[0], r[1]);
                    mma(low[1], s[ks].l, r[2], r[3]);
                    mma(m[0], s[ks].h, r[0], r[1]);
                    mma(m[1], s[ks].h, r[2], r[3]);
                }
                mma(low[0], s[ks].m, r[0], r[1]);
                mma(low[1], s[ks].m, r[2], r[3]);
            }
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) m[i][e] += low[i][e];
        };
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) split_tiles(S[2 * ks], S[2 * ks + 1], s[ks]);
        uint32_t th[4], tm[4], tl[4];
        load_matrix(c, TC_T, th, tm, tl);
        {
            float m[2][4];
            product(st + St::K, m);
#pragma unroll
            for (int i = 0; i < 2; ++i) *red_at(c & 1, 0, warp, i) = make_float4(m[i][0], m[i][1], m[i][2], m[i][3]);
        }
        __syncthreads();
        Parts p;
        fetch_x(c, p);
        float qs[2][4];
        product(st + St::Q, qs);                              // the tensor cores work on this while the partial sums arrive
        Split3 x;
        form_x(p, x);
        float u[2][4];
        times(x, th, tm, tl, u, Flag<true>());
        const float pc = f[3 * CK];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const float2 dk = *reinterpret_cast<const float2*>(f + 2 * CK + i * 8 + t4 * 2);
            u[i][0] *= dk.x;
            u[i][1] *= dk.y;
            u[i][2] *= dk.x;
            u[i][3] *= dk.y;
        }
        Split3 y;
        split_tiles(u[0], u[1], y);
#pragma unroll
        for (int i = 0; i < 2 * KS; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[i][e] *= pc;
        uint32_t r[KS][4];
#pragma unroll
        for (int ks = 0; ks < KS; ++ks)
            ldsm4t(r[ks], st + St::K + ((mi & 1) * 8 + mr) * St::PITCH + (d0 + ks * 16 + (mi >> 1) * 8) * 2);
#pragma unroll
        for (int i = 0; i < 2 * KS; ++i) mma(S[i], y.l, r[i >> 1][2 * (i & 1)], r[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
        for (int i = 0; i < 2 * KS; ++i) mma(S[i], y.m, r[i >> 1][2 * (i & 1)], r[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
        for (int i = 0; i < 2 * KS; ++i) mma(S[i], y.h, r[i >> 1][2 * (i & 1)], r[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
        for (int i = 0; i < 2; ++i) *red_at(c & 1, 1, warp, i) = make_float4(qs[i][0], qs[i][1], qs[i][2], qs[i][3]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2 * KS; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = d0 + i * 8 + t4 * 2 + (e & 1), col = gr + (e >> 1) * 8;
            if (d < dim && c0 + col < vdim) my_state[(size_t)d * vdim + col] = S[i][e];
        }
}

// ---- the scan on the FMA pipes (float32 rows, odd sizes) ----------------------------------------------------------------
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

constexpr int MAX_SMEM = 227 * 1024;

int sm_count() {
    static int n = 0;
    if (n == 0) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) n = 148;
    }
    return n;
}

// Shared memory that a scan's blocks ask for.  A block walks its sequence by itself, so a scan takes as long as its slowest block:
// several on one SM while others are idle (the kernel in front still fills them when blocks are handed out) would set the pace.
// Up to four rounds of blocks ask for so much that no SM takes more than its share.
size_t spread(long long blocks, size_t need) {
    const long long share = (blocks + sm_count() - 1) / sm_count();
    if (share > 4) return need;
    const size_t least = (size_t)(228 * 1024) / (size_t)(share + 1);
    return need > least ? need : least;
}

template <int KS>
int scan_tc(const void* q, const void* k, const void* v, long long ld, const void* rec, const int* seq_row0, const int* seq_len,
            const int* slots, float* state, long long slot_stride, float* out, long long ldo, int B, int H, int G, int dim, int vdim,
            cudaStream_t st) {
    const dim3 grid((vdim + 15) / 16, H, B);
    const size_t smem = spread((long long)grid.x * H * B, TcStage<KS>::TOTAL);
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(delta_scan_tc_kernel<KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM);
        set = true;
    }
    launch_pdl(delta_scan_tc_kernel<KS>, grid, dim3(TC_THREADS), smem, st, (const bf16*)q, (const bf16*)k, (const bf16*)v, ld,
               (const unsigned char*)rec, seq_row0, seq_len, slots, state, slot_stride, out, ldo, H, G, dim, vdim);
    QNN_LAUNCH_CHECK();
}

template <typename T, int RPT, int CPT, bool VEC>
int scan_as(const void* q, const void* k, const void* v, long long ld, const float* inv, int ldi, float q_scale, const float* rec,
            const int* seq_row0, const int* seq_len, const int* slots, float* state, long long slot_stride, float* out,
            long long ldo, int B, int H, int G, int dim, int vdim, cudaStream_t st) {
    using Buf = ScanBuf<RPT, CPT>;
    const dim3 grid((vdim + Buf::COLS - 1) / Buf::COLS, H, B);
    const size_t smem = spread((long long)grid.x * H * B, Buf::bytes(RPT <= 16 ? 2 : 1));
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(delta_scan_kernel<T, RPT, CPT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM);
        set = true;
    }
    launch_pdl(delta_scan_kernel<T, RPT, CPT, VEC>, grid, dim3(SCAN_THREADS), smem, st,
               (const T*)q, (const T*)k, (const T*)v, ld, inv, ldi, q_scale, rec, seq_row0, seq_len, slots, state, slot_stride, out,
               ldo, H, G, dim, vdim);
    QNN_LAUNCH_CHECK();
}

}  // namespace

// q, k: [rows, G * dim], v: [rows, H * vdim] of `dtype`, one row pitch `ld`; inv: [rows, ldi] with 1 / length of the G query heads,
// then of the G key heads; seq_row0, seq_len: first row and row count of the B sequences (both null: row b alone); pre:
// [rows, ldp] with b of the H heads, then a of the H heads; rate, bias: [H] float32 (rate = exp(A)); rec: at least (T / 16 + B) * H records of 3280 bytes (tensor_cores) or 544 floats.  longest: the most rows of a
// sequence.  dim up to 256.  tensor_cores: bfloat16 rows, dim and vdim multiples of 8, everything on 16 bytes.
QNN_API int qnn_delta_chunks(const void* q, const void* k, long long ld, int dtype, const float* inv, int ldi, const float* pre,
                             int ldp, const float* rate, const float* bias, float q_scale, const int* seq_row0, const int* seq_len,
                             void* rec, int B, int longest, int H, int G, int dim, int tensor_cores, cudaStream_t st) {
    if (B <= 0 || longest <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || dim <= 0 || dim > DELTA_MAX_DIM || B > 65535 || G > 65535 || ldi < 2 * G || ldp < 2 * H)
        return QNN_ERR_ARGUMENT;
    if ((seq_row0 == nullptr) != (seq_len == nullptr)) return QNN_ERR_ARGUMENT;
    if (tensor_cores) {
        if (dtype != QNN_DT_BF16 || dim % 8 || ld % 8 || (((uintptr_t)q | (uintptr_t)k | (uintptr_t)rec) & 15)) return QNN_ERR_ARGUMENT;
        const int dpad = (dim + 15) & ~15;
        const size_t smem = (size_t)4 * (2 * CK * (dpad * 2 + 16) + 3 * CK * (CK + 1) * 4);
        static bool set = false;
        if (!set) {
            cudaFuncSetAttribute(delta_chunks_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM);
            set = true;
        }
        launch_pdl(delta_chunks_tc_kernel, dim3((unsigned)((longest + 4 * CK - 1) / (4 * CK)), G, B), dim3(128), smem, st,
                   (const bf16*)q, (const bf16*)k, ld, inv, ldi, pre, ldp, rate, bias, q_scale, seq_row0, seq_len,
                   (unsigned char*)rec, H, G, dim);
        QNN_LAUNCH_CHECK();
    }
    const int pitch = ((dim + 3) & ~3) + 4;
    const size_t smem = ((size_t)2 * CK * pitch + 6 * CK * (CK + 1)) * sizeof(float);
    if (smem > 48 * 1024) return QNN_ERR_UNSUPPORTED;
    const dim3 grid((unsigned)((longest + CK - 1) / CK), G, B);
    if (dtype == QNN_DT_BF16)
        launch_pdl(delta_chunks_kernel<bf16>, grid, dim3(128), smem, st, (const bf16*)q, (const bf16*)k, ld, inv, ldi, pre, ldp,
                   rate, bias, q_scale, seq_row0, seq_len, (float*)rec, H, G, dim);
    else
        launch_pdl(delta_chunks_kernel<float>, grid, dim3(128), smem, st, (const float*)q, (const float*)k, ld, inv, ldi, pre, ldp,
                   rate, bias, q_scale, seq_row0, seq_len, (float*)rec, H, G, dim);
    QNN_LAUNCH_CHECK();
}

// The same rows; slots: the state slot of each sequence (negative: nothing is read or written); state: slot s's
// [H, dim, vdim] floats at state + s * slot_stride; out: [rows, ldo] float32, H * vdim columns; cpt: 16 or 32 value columns per
// block (1 or 2: many sequences fill the device with the wider ones, which read the rows half as often).  tensor_cores: rec as
// qnn_delta_chunks left it with the same; cpt, inv and q_scale are not read then.
QNN_API int qnn_delta_scan(const void* q, const void* k, const void* v, long long ld, int dtype, const float* inv, int ldi,
                           float q_scale, const void* rec_, const int* seq_row0, const int* seq_len, const int* slots, float* state,
                           long long slot_stride, float* out, long long ldo, int B, int H, int G, int dim, int vdim, int cpt,
                           int tensor_cores,
                           cudaStream_t st) {
    if (B <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || dim <= 0 || dim > DELTA_MAX_DIM || vdim <= 0 || B > 65535 || H > 65535 || ldi < 2 * G ||
        slot_stride < (long long)H * dim * vdim || (cpt != 1 && cpt != 2) || (seq_row0 == nullptr) != (seq_len == nullptr))
        return QNN_ERR_ARGUMENT;
    const size_t es = dtype == QNN_DT_BF16 ? 2 : 4;
    const bool vec = dim % 8 == 0 && vdim % 8 == 0 && (ld * es) % 16 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15) == 0;
    if (tensor_cores) {
        if (dtype != QNN_DT_BF16 || !vec || ((uintptr_t)rec_ & 15)) return QNN_ERR_ARGUMENT;
        if (dim <= 64) return scan_tc<1>(q, k, v, ld, rec_, seq_row0, seq_len, slots, state, slot_stride, out, ldo, B, H, G, dim, vdim, st);
        if (dim <= 128) return scan_tc<2>(q, k, v, ld, rec_, seq_row0, seq_len, slots, state, slot_stride, out, ldo, B, H, G, dim, vdim, st);
        return scan_tc<4>(q, k, v, ld, rec_, seq_row0, seq_len, slots, state, slot_stride, out, ldo, B, H, G, dim, vdim, st);
    }
    const float* rec = (const float*)rec_;
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
    if (dtype == QNN_DT_BF16) {                               // (aligned bfloat16 rows have the tensor-core kernel)
        QNN_DS_ROWS(bf16, false)
    } else {
        if (vec) { QNN_DS_ROWS(float, true) } else { QNN_DS_ROWS(float, false) }
    }
#undef QNN_DS_ROWS
#undef QNN_DS_COLS
#undef QNN_DS
}
