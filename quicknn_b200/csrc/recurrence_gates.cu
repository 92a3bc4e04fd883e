// The gates of a real-gated linear recurrence for many rows, and the first pass over its segments, in one kernel (what this
// leaves is described at the head of linear_recurrence.cu; the formulas are those of its `gates`).
//
// A CTA owns 64 rows (two segments of 32) of one sequence and 64 channels of one part.  The product is that of
// block_linear.cu: u of the part against the r rows and the i rows of the channels, 64 x 128 outputs, mma.sync m16n8k16, a
// cp.async ring of two stages of 64 inner elements, float32 sums.  The logits stay in shared memory; then a thread per
// channel and segment forms (a, term) of its rows in order, writes them out and leaves the segment's product of a and the
// state that it reaches.
#include "common.cuh"

using namespace qnn;

namespace {

__device__ __forceinline__ void cp_async_16(unsigned dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;       // 0 source bytes: the destination is zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr int BM = 64, CH = 64, BN = 2 * CH, BK = 64, STAGES = 2, THREADS = 128, ROWB = BK * 2;   // four CTAs per SM
constexpr int SEG = 32, STAGE = (BM + BN) * ROWB, LDL = BN + 1;
constexpr size_t SMEM = (size_t)STAGES * STAGE;
static_assert((size_t)BM * LDL * 4 <= SMEM, "the logits take the ring's place");
static_assert(THREADS == CH * (BM / SEG), "a thread per channel and segment");

// 32-bit arithmetic on the fast exponential, quotient and square root (relative errors of about 1e-6; u and the product's
// operands are bfloat16).
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
// 1 - e^t for t <= 0, with the digits kept where t is near 0 (there the Taylor sum, remainder below 3e-7 of it)
__device__ __forceinline__ float one_minus_exp(float t) {
    const float series = -t * fmaf(t * 0.5f, fmaf(t * (1.f / 3.f), fmaf(t * 0.25f, fmaf(t * 0.2f, fmaf(t, 1.f / 6.f, 1.f), 1.f), 1.f), 1.f), 1.f);
    return t > -0.35f ? series : 1.f - __expf(t);
}
__device__ __forceinline__ float sqrt_fast(float x) {
    float r;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}

struct Gates {
    const bf16* u;              // rows of pitch ldu
    const bf16* w;              // [blocks][r rows, i rows][part]
    const float* rb;
    const float* ib;
    const float* decay;
    float* z;                   // rows of pitch ldz: per part first a, then the term
    const float* state;         // slot s: state + s * slot_stride
    float* scratch;             // [sequences][nseg][3][C]
    const int* seq_row0;
    const int* seq_len;
    const int* slots;
    long long ldu, ldz, slot_stride;
    int C, part, nseg, tiles;   // tiles: channel tiles of a part
};

__global__ void __launch_bounds__(THREADS, 4) recurrence_gates_kernel(const Gates p) {
    extern __shared__ __align__(128) unsigned char smem[];
    float* logits = reinterpret_cast<float*>(smem);             // [BM][LDL], once the products are done
    const int blk = blockIdx.x / p.tiles, c0 = (blockIdx.x - blk * p.tiles) * CH;
    const int b = blockIdx.z, m0 = blockIdx.y * BM;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int wm = warp >> 1, wn = warp & 1;                    // warp tiles of 32 x 64
    const int n = p.seq_len[b], slot = p.slots[b];              // from the host, before the step
    if (m0 >= n || slot < 0) return;
    const int row0 = p.seq_row0[b] + m0, rows = min(BM, n - m0);
    const bf16* ub = p.u + (size_t)row0 * p.ldu + (size_t)blk * p.part;
    const bf16* wb = p.w + (size_t)blk * 2 * p.part * p.part;
    const unsigned base = (unsigned)__cvta_generic_to_shared(smem);
    const int nk = (p.part + BK - 1) / BK;
    auto load_w = [&](int kb) {
        const unsigned sb = base + (kb % STAGES) * STAGE + BM * ROWB;
#pragma unroll
        for (int i = tid; i < BN * 8; i += THREADS) {
            const int r = i >> 3, c = i & 7, k = kb * BK + c * 8, ch = c0 + (r & (CH - 1));
            const bool ok = ch < p.part && k < p.part;
            const bf16* src = ok ? wb + (size_t)((r < CH ? 0 : p.part) + ch) * p.part + k : p.w;
            cp_async_16(sb + r * ROWB + ((c ^ (r & 7)) << 4), src, ok);
        }
    };
    auto load_u = [&](int kb) {
        const unsigned sa = base + (kb % STAGES) * STAGE;
#pragma unroll
        for (int i = tid; i < BM * 8; i += THREADS) {
            const int r = i >> 3, c = i & 7, k = kb * BK + c * 8;
            const bool ok = r < rows && k < p.part;
            cp_async_16(sa + r * ROWB + ((c ^ (r & 7)) << 4), ok ? ub + (size_t)r * p.ldu + k : p.u, ok);
        }
    };
    // weights are written by no kernel: the first stages' ask for them before the wait for the kernel in front
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s)
        if (s < nk) load_w(s);
    pdl_wait();
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) {
        if (s < nk) load_u(s);
        cp_async_commit();                                      // (the first group also holds the weights asked for above)
    }
    float acc[2][8][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
    for (int kb = 0; kb < nk; ++kb) {
        cp_async_wait<STAGES - 2>();
        __syncthreads();
        if (kb + STAGES - 1 < nk) {
            load_w(kb + STAGES - 1);
            load_u(kb + STAGES - 1);
        }
        cp_async_commit();
        const unsigned sa = base + (kb % STAGES) * STAGE, sb = sa + BM * ROWB;
#pragma unroll
        for (int ks = 0; ks < BK / 16; ++ks) {
            uint32_t af[2][4], bf[4][4];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int r = wm * 32 + i * 16 + (lane & 15), c = ks * 2 + (lane >> 4);
                ldmatrix_x4(af[i], sa + r * ROWB + ((c ^ (r & 7)) << 4));
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int r = wn * 64 + j * 16 + (lane & 7) + ((lane >> 4) << 3), c = ks * 2 + ((lane >> 3) & 1);
                ldmatrix_x4(bf[j], sb + r * ROWB + ((c ^ (r & 7)) << 4));
            }
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    mma_16816(acc[i][2 * j], af[i], bf[j][0], bf[j][1]);
                    mma_16816(acc[i][2 * j + 1], af[i], bf[j][2], bf[j][3]);
                }
        }
    }
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                logits[(wm * 32 + i * 16 + g + (e >> 1) * 8) * LDL + wn * 64 + j * 8 + t4 * 2 + (e & 1)] = acc[i][j][e];
    __syncthreads();
    const int cl = tid & (CH - 1), seg = tid / CH, k = c0 + cl;
    const int r0 = seg * SEG, r1 = min(r0 + SEG, rows);
    if (k >= p.part || r0 >= rows) return;
    const int ch = blk * p.part + k;
    const float br = p.rb[ch], bi = p.ib[ch], decay = p.decay[ch];
    float* sc = p.scratch + ((size_t)b * p.nseg + (m0 + r0) / SEG) * 3 * p.C + ch;
    float S = 0.f, all = 1.f;
    if (m0 + r0 == 0) {
        S = p.state[(size_t)slot * p.slot_stride + ch];
        sc[2 * (size_t)p.C] = S;
    }
    const bf16* uc = ub + (size_t)r0 * p.ldu + k;
    float* zc = p.z + (size_t)(row0 + r0) * p.ldz + (size_t)blk * 2 * p.part + k;
    const float* lg = logits + r0 * LDL + cl;
    auto row = [&](float u, int i) {                            // row r0 + i of the segment
        const float la = -decay * sigmoid_fast(lg[i * LDL] + br);
        const float a = __expf(la), term = sqrt_fast(one_minus_exp(2.f * la)) * sigmoid_fast(lg[i * LDL + CH] + bi) * u;
        zc[0] = a;
        zc[p.part] = term;
        zc += p.ldz;
        all *= a;
        S = fmaf(a, S, term);
    };
    if (r1 - r0 == SEG) {
        constexpr int AHEAD = 16;                               // rows of u asked for together
#pragma unroll 1
        for (int r = 0; r < SEG; r += AHEAD) {
            bf16 u[AHEAD];
#pragma unroll
            for (int i = 0; i < AHEAD; ++i) u[i] = uc[(size_t)i * p.ldu];
            uc += (size_t)AHEAD * p.ldu;
#pragma unroll
            for (int i = 0; i < AHEAD; ++i) row(__bfloat162float(u[i]), i);
            lg += AHEAD * LDL;
        }
    } else {
        for (int r = 0; r < r1 - r0; ++r) row(__bfloat162float(uc[(size_t)r * p.ldu]), r);
    }
    sc[0] = all;
    sc[p.C] = S;
}

}  // namespace

// u, w: bfloat16.  z: [rows, 2C] float32, scratch: n_seqs * nseg * 3 * C floats, segments of 32 rows: what
// qnn_linear_recurrence takes with gates_done.  seq_len and slots are read before the wait for the kernel in front on the
// stream: that kernel must not be the one that writes them.
QNN_API int qnn_recurrence_gates(const void* u, long long ldu, const void* w, const float* rb, const float* ib, const float* decay,
                                 float* z, long long ldz, const float* state, long long slot_stride, float* scratch,
                                 const int* seq_row0, const int* seq_len, const int* slots, int n_seqs, int longest, int C,
                                 int part, int nseg, cudaStream_t st) {
    if (n_seqs <= 0 || longest <= 0) return 0;
    if (C <= 0 || part <= 0 || C % part || ldu < C || ldz < 2LL * C || slot_stride < C || nseg < (longest + SEG - 1) / SEG ||
        seq_row0 == nullptr || seq_len == nullptr || scratch == nullptr)
        return QNN_ERR_ARGUMENT;
    const long long y = (longest + BM - 1) / BM;
    if (part % 8 || ldu % 8 || (((uintptr_t)u | (uintptr_t)w) & 15) || y > 65535 || n_seqs > 65535) return QNN_ERR_UNSUPPORTED;
    Gates p;
    p.u = (const bf16*)u; p.w = (const bf16*)w; p.rb = rb; p.ib = ib; p.decay = decay; p.z = z; p.state = state;
    p.scratch = scratch; p.seq_row0 = seq_row0; p.seq_len = seq_len; p.slots = slots; p.ldu = ldu; p.ldz = ldz;
    p.slot_stride = slot_stride; p.C = C; p.part = part; p.nseg = nseg; p.tiles = (part + CH - 1) / CH;
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(recurrence_gates_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    launch_pdl(recurrence_gates_kernel, dim3((unsigned)(p.tiles * (C / part)), (unsigned)y, n_seqs), dim3(THREADS), SMEM, st, p);
    QNN_LAUNCH_CHECK();
}
