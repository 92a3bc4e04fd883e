// Block-diagonal products: rows cut into equal parts, each part times a matrix of its own.
//
//   qnn_block_linear   out[t, b, :] = W_b x[t, b, :]       W: [blocks, N, K];  optionally times sigmoid(gate[t, b, :])
//
// The parts of x lie `x_step` columns apart in rows of pitch ldx; part b of the result is columns b * N .. of rows of pitch
// ldo.  bfloat16 or float32 in, bfloat16 or float32 out, float32 sums in the order of the inner size, so a row's result does
// not depend on which other rows share its tile.  Used for the gates of a linear recurrence (float32 out: what enters the
// recurrence is not rounded) and for values that every head forms from one latent.
//
// Kernels: bfloat16 with inner sizes and pitches in whole 16-byte pieces on the tensor cores (mma.sync m16n8k16, tiles of
// 128 x 128, 64 x 64, 16 x 64 or 16 x 32, a cp.async ring of three to eight stages of 64 inner elements, 16-byte chunks XOR-ed
// with the row number); everything else on a plain FMA kernel, 32 x 32 tiles.
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

struct Args {
    const void* x;
    const void* w;
    void* out;
    const void* gate;           // null, or rows of pitch ldg whose column b * N + n gates that output
    long long ldx, x_step, ldo, ldg;
    int x_dt, w_dt, out_dt, gate_dt, T, N, K;
};

__device__ __forceinline__ float gated(const Args& a, int t, size_t col, float v) {
    if (a.gate == nullptr) return v;
    const float z = load_as_f(a.gate, a.gate_dt, (size_t)t * a.ldg + col);
    return v * (1.f / (1.f + expf(-z)));
}

// BM x BN tile of one block's product, WM x WN warps, each (BM / WM) x (BN / WN); BK = 64 inner elements per stage.
template <int BM, int BN, int WM, int WN, int STAGES>
__global__ void __launch_bounds__(WM * WN * 32)
block_linear_mma_kernel(const Args a) {
    constexpr int BK = 64, THREADS = WM * WN * 32, ROWB = BK * 2;
    constexpr int TM = BM / WM, TN = BN / WN, MT = TM / 16, NT = TN / 8;
    static_assert(TM % 16 == 0 && TN % 16 == 0, "warp tiles are made of 16 x 16 pieces");
    constexpr int STAGE = (BM + BN) * ROWB;
    extern __shared__ __align__(128) unsigned char smem[];
    pdl_wait();
    const int b = blockIdx.z, n0 = blockIdx.x * BN, m0 = blockIdx.y * BM;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int wm = warp / WN, wn = warp % WN;
    const bf16* xb = (const bf16*)a.x + (size_t)b * a.x_step;
    const bf16* wb = (const bf16*)a.w + (size_t)b * a.N * a.K;
    const unsigned base = (unsigned)__cvta_generic_to_shared(smem);
    const int nk = (a.K + BK - 1) / BK;
    auto load = [&](int kb) {
        if (kb < nk) {
            const unsigned sa = base + (kb % STAGES) * STAGE, sb = sa + BM * ROWB;
            for (int i = tid; i < BM * 8; i += THREADS) {
                const int r = i >> 3, c = i & 7, k = kb * BK + c * 8;
                const bool ok = m0 + r < a.T && k < a.K;
                cp_async_16(sa + r * ROWB + ((c ^ (r & 7)) << 4), ok ? (const void*)(xb + (size_t)(m0 + r) * a.ldx + k) : a.x, ok);
            }
            for (int i = tid; i < BN * 8; i += THREADS) {
                const int r = i >> 3, c = i & 7, k = kb * BK + c * 8;
                const bool ok = n0 + r < a.N && k < a.K;
                cp_async_16(sb + r * ROWB + ((c ^ (r & 7)) << 4), ok ? (const void*)(wb + (size_t)(n0 + r) * a.K + k) : a.w, ok);
            }
        }
        cp_async_commit();
    };
    float acc[MT][NT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) load(s);
    for (int kb = 0; kb < nk; ++kb) {
        cp_async_wait<STAGES - 2>();
        __syncthreads();
        load(kb + STAGES - 1);                    // refills the stage that the round before read
        const unsigned sa = base + (kb % STAGES) * STAGE, sb = sa + BM * ROWB;
#pragma unroll
        for (int ks = 0; ks < BK / 16; ++ks) {
            uint32_t af[MT][4], bfr[NT / 2][4];
#pragma unroll
            for (int i = 0; i < MT; ++i) {
                const int r = wm * TM + i * 16 + (lane & 15), c = ks * 2 + (lane >> 4);
                ldmatrix_x4(af[i], sa + r * ROWB + ((c ^ (r & 7)) << 4));
            }
#pragma unroll
            for (int j = 0; j < NT / 2; ++j) {
                const int r = wn * TN + j * 16 + (lane & 7) + ((lane >> 4) << 3), c = ks * 2 + ((lane >> 3) & 1);
                ldmatrix_x4(bfr[j], sb + r * ROWB + ((c ^ (r & 7)) << 4));
            }
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int j = 0; j < NT / 2; ++j) {
                    mma_16816(acc[i][2 * j], af[i], bfr[j][0], bfr[j][1]);
                    mma_16816(acc[i][2 * j + 1], af[i], bfr[j][2], bfr[j][3]);
                }
        }
    }
    const bool pair = ((a.N | a.ldo) & 1) == 0;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int t = m0 + wm * TM + i * 16 + g + h * 8;
            if (t >= a.T) continue;
            float z[NT][2];
            if (a.gate != nullptr) {                  // the row's gates are asked for together
                const size_t at = (size_t)t * a.ldg + (size_t)b * a.N;
                if (a.gate_dt == QNN_DT_BF16) {
                    bf16 raw[NT][2];
#pragma unroll
                    for (int j = 0; j < NT; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) raw[j][e] = ((const bf16*)a.gate)[at + min(n0 + wn * TN + j * 8 + t4 * 2 + e, a.N - 1)];
#pragma unroll
                    for (int j = 0; j < NT; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) z[j][e] = __bfloat162float(raw[j][e]);
                } else {
#pragma unroll
                    for (int j = 0; j < NT; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) z[j][e] = ((const float*)a.gate)[at + min(n0 + wn * TN + j * 8 + t4 * 2 + e, a.N - 1)];
                }
            }
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int n = n0 + wn * TN + j * 8 + t4 * 2;
                if (n >= a.N) continue;
                const size_t col = (size_t)b * a.N + n;
                float v0 = acc[i][j][2 * h], v1 = acc[i][j][2 * h + 1];
                if (a.gate != nullptr) {
                    v0 *= __fdividef(1.f, 1.f + __expf(-z[j][0]));
                    v1 *= __fdividef(1.f, 1.f + __expf(-z[j][1]));
                }
                const size_t at = (size_t)t * a.ldo + col;
                if (pair) {
                    if (a.out_dt == QNN_DT_BF16) *reinterpret_cast<__nv_bfloat162*>((bf16*)a.out + at) = __floats2bfloat162_rn(v0, v1);
                    else *reinterpret_cast<float2*>((float*)a.out + at) = make_float2(v0, v1);
                } else {
                    store_from_f(a.out, a.out_dt, at, v0);
                    if (n + 1 < a.N) store_from_f(a.out, a.out_dt, at + 1, v1);
                }
            }
        }
}

// 32 x 32 outputs per block of 256 threads (four rows each), 32 inner elements at a time through shared memory.
__global__ void __launch_bounds__(256) block_linear_kernel(const Args a) {
    __shared__ float xs[32][33], ws[32][33];
    pdl_wait();
    const int b = blockIdx.z, n0 = blockIdx.x * 32, m0 = blockIdx.y * 32;
    const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < a.K; k0 += 32) {
        __syncthreads();
        for (int i = ty; i < 32; i += 8) {
            const int k = k0 + tx;
            xs[i][tx] = (m0 + i < a.T && k < a.K) ? load_as_f(a.x, a.x_dt, (size_t)(m0 + i) * a.ldx + (size_t)b * a.x_step + k) : 0.f;
            ws[i][tx] = (n0 + i < a.N && k < a.K) ? load_as_f(a.w, a.w_dt, ((size_t)b * a.N + n0 + i) * a.K + k) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < 32; ++k) {
            const float wv = ws[tx][k];
#pragma unroll
            for (int q = 0; q < 4; ++q) acc[q] = fmaf(xs[ty + q * 8][k], wv, acc[q]);
        }
    }
    const int n = n0 + tx;
    if (n >= a.N) return;
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        const int t = m0 + ty + q * 8;
        if (t < a.T) {
            const size_t col = (size_t)b * a.N + n;
            store_from_f(a.out, a.out_dt, (size_t)t * a.ldo + col, gated(a, t, col, acc[q]));
        }
    }
}

template <int BM, int BN, int WM, int WN, int STAGES>
int launch_mma(const Args& a, int blocks, cudaStream_t st) {
    auto kern = block_linear_mma_kernel<BM, BN, WM, WN, STAGES>;
    constexpr size_t smem = (size_t)STAGES * (BM + BN) * 128;
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const dim3 grid((a.N + BN - 1) / BN, (a.T + BM - 1) / BM, blocks);
    launch_pdl(kern, grid, dim3(WM * WN * 32), smem, st, a);
    return (int)cudaGetLastError();
}

}  // namespace

QNN_API int qnn_block_linear(const void* x, int x_dt, long long ldx, long long x_step, const void* w, int w_dt, void* out,
                             int out_dt, long long ldo, const void* gate, int gate_dt, long long ldg, int T, int blocks, int N,
                             int K, cudaStream_t st) {
    if (T <= 0 || blocks <= 0) return 0;
    if (N <= 0 || K <= 0 || blocks > 65535 || ldo < (long long)blocks * N || ldx < (long long)(blocks - 1) * x_step + K) return QNN_ERR_ARGUMENT;
    if ((T + 15) / 16 > 65535) return QNN_ERR_UNSUPPORTED;
    Args a;
    a.x = x; a.w = w; a.out = out; a.gate = gate; a.ldx = ldx; a.x_step = x_step; a.ldo = ldo; a.ldg = ldg;
    a.x_dt = x_dt; a.w_dt = w_dt; a.out_dt = out_dt; a.gate_dt = gate_dt; a.T = T; a.N = N; a.K = K;
    const bool tensor = x_dt == QNN_DT_BF16 && w_dt == QNN_DT_BF16 && K % 8 == 0 && ldx % 8 == 0 && x_step % 8 == 0 &&
                        (((uintptr_t)x | (uintptr_t)w) & 15) == 0 && ((uintptr_t)out & 7) == 0;
    if (tensor) {
        if (T <= 32) return launch_mma<16, 64, 1, 4, 3>(a, blocks, st);
        // a few outputs of a long inner size: blocks of 16 rows fill the device, with eight stages on their way
        if (blocks == 1 && N <= 32) return launch_mma<16, 32, 1, 2, 8>(a, blocks, st);
        if (blocks == 1 && N <= 64) return launch_mma<16, 64, 1, 4, 8>(a, blocks, st);
        const long long big = (long long)((T + 127) / 128) * ((N + 127) / 128) * blocks;
        if (N > 64 && big >= 448) return launch_mma<128, 128, 2, 4, 3>(a, blocks, st);
        return launch_mma<64, 64, 2, 2, 3>(a, blocks, st);
    }
    launch_pdl(block_linear_kernel, dim3((N + 31) / 32, (T + 31) / 32, blocks), dim3(256), 0, st, a);
    QNN_LAUNCH_CHECK();
}
