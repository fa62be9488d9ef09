// Linear attention with a fixed decay per head (retention and its kin) on the packed-step layout of seq_ops.cu: a matrix
// S [D, E] per head and request,
//
//     S_t = decay_h S_(t-1) + k_t v_t^T,      o_t = S_t^T q_t
//
// no softmax, no denominator. q, k and v come straight out of the fused projection (fp32 columns of src) and are brought
// into shape on their way to shared memory: rotary positions on q and k from a table of the step's cosines and sines
// (llark_seq_rotary_table), a factor on k, or SiLU on all three. Everything is fp32: positions and angles, q / k / v, the
// decays, the state and the outputs.
//
//   llark_seq_rotary_table   cos / sin of position * frequency for every row of the step (one table serves every layer, head
//                            and pass with the same frequencies)
//   llark_seq_decay_rows     the recurrence token by token with the state in registers, coalesced state reads and writes:
//                            single-token steps, short portions, any head size up to 1024, and the all-fp32 mode
//   llark_seq_decay_chunks   prompts: 32 tokens at a time as matrix products on the tensor cores,
//                                A = (Q K^T) .* decay^(i-j) (j <= i),   O = decay^(i+1) Q S + A V,   S = decay^n S + (decay^(n-1-j) K)^T V
//                            every product in three TF32 products of split operands (x = hi + lo, dropping lo * lo), which
//                            keeps fp32 accuracy (2^-21 relative); the state stays in accumulator registers, transposed, so
//                            that a fragment of it is directly the B operand of Q S. Long prompts run as chunks in three
//                            passes (local states from zero, llark_seq_decay_combine, outputs) to fill the GPU.
#include "common.cuh"

namespace llark {
extern thread_local int g_last_cuda_error;
namespace decay {

static int check_launch() {
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) {
        g_last_cuda_error = (int)e;
        return LLARK_ECUDA;
    }
    return LLARK_OK;
}

__device__ __forceinline__ float siluf_(float z) { return z / (1.0f + expf(-z)); }

__global__ void rotary_table_kernel(const float* __restrict__ freq, int n_freq, const int* __restrict__ tok_seq,
                                    const int* __restrict__ cu, const int* __restrict__ pos0, float2* __restrict__ cs,
                                    int n_tok) {
    const long long n = (long long)n_tok * n_freq;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const int t = (int)(i / n_freq), f = (int)(i % n_freq);
        const int b = tok_seq[t];
        float s, c;
        sincosf((float)(pos0[b] + (t - cu[b])) * freq[f], &s, &c);
        cs[i] = make_float2(c, s);
    }
}

// Where a step's q, k and v are and what is done to them on the way in.
struct DecayIn {
    const float* src;
    long long ld;
    int q_off, k_off, v_off;
    const float2* cs;  // [n_tok, n_rot / 2] cosines and sines, NULL without rotation
    int n_rot, interleaved;
    float k_scale;
    int silu;
};

// entry d of a q or k head of row t (x = the head's first entry)
__device__ __forceinline__ float qk_entry(const DecayIn& in, const float* x, long long t, int d) {
    float v = x[d];
    if (in.silu) return siluf_(v);
    if (d < in.n_rot) {
        const int half = in.n_rot >> 1;
        const int i = in.interleaved ? d >> 1 : (d < half ? d : d - half);
        const bool second = in.interleaved ? (d & 1) : d >= half;
        const float w = x[in.interleaved ? d ^ 1 : (second ? i : i + half)];
        const float2 c = in.cs[t * half + i];
        v = second ? v * c.x + w * c.y : v * c.x - w * c.y;
    }
    return v;
}

// ------------------------------------------------------------------------------------------------ token by token
// Block = 32 columns of one head of one work item (a run of rows of one request, see seq_mixers.cu). Lane l of a warp holds
// four adjacent columns (l % 8) of the rows rg + 32 i, rg = 4 * warp + l / 8: a warp reads and writes the state in 128-byte
// row pieces. A tile of ts tokens is brought to shared memory, each token then needs one shuffle over the four row groups
// of a warp; the eight warps' partial outputs are added up once per tile.
template <int RPT>
__global__ void __launch_bounds__(256)
decay_rows_kernel(DecayIn in, const float* __restrict__ pow_h, int pow_ld, const float* __restrict__ init_buf,
                  float* __restrict__ final_buf, float* __restrict__ o, const int* __restrict__ item_row0,
                  const int* __restrict__ item_n, const int* __restrict__ item_init, const int* __restrict__ item_final, int H,
                  int D, int E, int ts, int vec) {
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;                  // [ts][D]
    float* sk = sq + ts * D;         // [ts][D]
    float* sv = sk + ts * D;         // [ts][32]  (ts * D is rounded up to a multiple of 4 by the launcher's choice of ts)
    float* part = sv + ts * 32;      // [ts][8][32]
    const int h = blockIdx.y, b = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c4 = (lane & 7) * 4, rg = warp * 4 + (lane >> 3);
    const int e0 = blockIdx.x * 32;
    const int row0 = item_row0[b], n = item_n[b];
    const float dec = pow_h[(long long)h * pow_ld + 1];
    float S[RPT][4];
    const long long de = (long long)D * E;
    const float* si = item_init[b] >= 0 ? init_buf + ((long long)item_init[b] * H + h) * de : nullptr;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = rg + 32 * i;
        S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
        if (si && d < D) {
            const float* p = si + (long long)d * E + e0 + c4;
            if (vec && e0 + c4 + 3 < E) {
                const float4 v = *reinterpret_cast<const float4*>(p);
                S[i][0] = v.x, S[i][1] = v.y, S[i][2] = v.z, S[i][3] = v.w;
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (e0 + c4 + c < E) S[i][c] = p[c];
            }
        }
    }
    for (int t0 = 0; t0 < n; t0 += ts) {
        const int cnt = n - t0 < ts ? n - t0 : ts;
        for (int i = threadIdx.x; i < cnt * D; i += 256) {
            const int tk = i / D, d = i % D;
            const long long t = row0 + t0 + tk;
            const float* r = in.src + t * in.ld + (long long)h * D;
            sq[i] = qk_entry(in, r + in.q_off, t, d);
            sk[i] = qk_entry(in, r + in.k_off, t, d) * in.k_scale;
        }
        for (int i = threadIdx.x; i < cnt * 32; i += 256) {
            const int tk = i >> 5, c = i & 31;
            float v = 0.f;
            if (e0 + c < E) {
                v = in.src[(long long)(row0 + t0 + tk) * in.ld + in.v_off + (long long)h * E + e0 + c];
                if (in.silu) v = siluf_(v);
            }
            sv[i] = v;
        }
        __syncthreads();
        for (int tk = 0; tk < cnt; ++tk) {
            float v[4], os[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int c = 0; c < 4; ++c) v[c] = sv[tk * 32 + c4 + c];
#pragma unroll
            for (int i = 0; i < RPT; ++i) {
                const int d = rg + 32 * i;
                const float kd = d < D ? sk[tk * D + d] : 0.f, qd = d < D ? sq[tk * D + d] : 0.f;
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    S[i][c] = fmaf(kd, v[c], dec * S[i][c]);
                    os[c] = fmaf(qd, S[i][c], os[c]);
                }
            }
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                os[c] += __shfl_xor_sync(0xffffffffu, os[c], 8);
                os[c] += __shfl_xor_sync(0xffffffffu, os[c], 16);
                if (lane < 8) part[(tk * 8 + warp) * 32 + c4 + c] = os[c];
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < cnt * 32; i += 256) {
            const int tk = i >> 5, c = i & 31;
            float s = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) s += part[(tk * 8 + w) * 32 + c];
            if (e0 + c < E) o[(long long)(row0 + t0 + tk) * H * E + (long long)h * E + e0 + c] = s;
        }
    }
    if (item_final[b] < 0) return;
    float* sf = final_buf + ((long long)item_final[b] * H + h) * de;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = rg + 32 * i;
        if (d < D) {
            float* p = sf + (long long)d * E + e0 + c4;
            if (vec && e0 + c4 + 3 < E) {
                *reinterpret_cast<float4*>(p) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (e0 + c4 + c < E) p[c] = S[i][c];
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ 32 tokens at a time
constexpr int kL = 32;        // tokens per block of products
constexpr int kAS = kL + 4;   // row pitch of A in shared memory

// x = hi + lo + (what neither holds, < 2^-21 |x|), both representable in TF32
__device__ __forceinline__ void split(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi)) & 0xffffe000u;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct FragA {
    uint32_t hi[4], lo[4];
    __device__ __forceinline__ void set(float x0, float x1, float x2, float x3) {
        split(x0, hi[0], lo[0]);
        split(x1, hi[1], lo[1]);
        split(x2, hi[2], lo[2]);
        split(x3, hi[3], lo[3]);
    }
};
struct FragB {
    uint32_t hi[2], lo[2];
    __device__ __forceinline__ void set(float x0, float x1) {
        split(x0, hi[0], lo[0]);
        split(x1, hi[1], lo[1]);
    }
};
__device__ __forceinline__ void mma3(float (&c)[4], const FragA& a, const FragB& b) {
    mma_tf32(c, a.lo, b.hi[0], b.hi[1]);
    mma_tf32(c, a.hi, b.lo[0], b.lo[1]);
    mma_tf32(c, a.hi, b.hi[0], b.hi[1]);
}

// Rows of one head (D entries from column off of src) -> dst [kL][pitch], zero behind the step's rows and behind D, as
// asynchronous copies of 16 bytes (vec) or of single words.
__device__ __forceinline__ void copy16(float* dst, const float* src, bool live) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy4(float* dst, const float* src, bool live) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 4 : 0) : "memory");
}
__device__ __forceinline__ void fetch_head(const float* src, long long ld, int cnt, int D, int Dp, int pitch, int vec, float* dst) {
    if (vec) {
        const int nq = Dp >> 2;
        for (int i = threadIdx.x; i < kL * nq; i += blockDim.x) {
            const int tk = i / nq, d = (i % nq) * 4;
            const bool live = tk < cnt && d < D;
            copy16(dst + tk * pitch + d, live ? src + tk * ld + d : src, live);
        }
    } else {
        for (int i = threadIdx.x; i < kL * Dp; i += blockDim.x) {
            const int tk = i / Dp, d = i % Dp;
            const bool live = tk < cnt && d < D;
            copy4(dst + tk * pitch + d, live ? src + tk * ld + d : src, live);
        }
    }
}
// SiLU in the accuracy of the fast exponential and division (about 2^-21 relative), in place over kL rows
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ void silu_rows(float* x, int width, int pitch) {
    const int nq = width >> 2;
    for (int i = threadIdx.x; i < kL * nq; i += blockDim.x) {
        float4* p = reinterpret_cast<float4*>(x + (i / nq) * pitch + (i % nq) * 4);
        const float4 v = *p;
        *p = make_float4(silu_fast(v.x), silu_fast(v.y), silu_fast(v.z), silu_fast(v.w));
    }
}
__device__ __forceinline__ void turn4(float4& u, float4& v, float4 c0, float4 c1, float f) {
    const float4 a = u, b = v;  // c0, c1: (cos, sin) of four neighbouring pairs (u.x, v.x) .. (u.w, v.w)
    u = make_float4((a.x * c0.x - b.x * c0.y) * f, (a.y * c0.z - b.y * c0.w) * f, (a.z * c1.x - b.z * c1.y) * f,
                    (a.w * c1.z - b.w * c1.w) * f);
    v = make_float4((b.x * c0.x + a.x * c0.y) * f, (b.y * c0.z + a.y * c0.w) * f, (b.z * c1.x + a.z * c1.y) * f,
                    (b.w * c1.z + a.w * c1.w) * f);
}
// Rotation of q (when there is one) and k and the factor on k, in place. A pair belongs to one thread.
__device__ __forceinline__ void turn_rows(const DecayIn& in, long long row, int cnt, int D, int DS, float* sQ, float* sK) {
    const int half = in.n_rot >> 1;
    const float f = in.k_scale;
    if (half && half % 4 == 0 && !in.interleaved) {
        const int nq = half >> 2;
        for (int i = threadIdx.x; i < cnt * nq; i += blockDim.x) {
            const int tk = i / nq, d = (i % nq) * 4;
            const float4* cp = reinterpret_cast<const float4*>(in.cs + (row + tk) * half + d);
            const float4 c0 = __ldg(cp), c1 = __ldg(cp + 1);
            float4* ku = reinterpret_cast<float4*>(sK + tk * DS + d);
            float4* kv = reinterpret_cast<float4*>(sK + tk * DS + d + half);
            float4 u = *ku, v = *kv;
            turn4(u, v, c0, c1, f);
            *ku = u, *kv = v;
            if (sQ) {
                float4* qu = reinterpret_cast<float4*>(sQ + tk * DS + d);
                float4* qv = reinterpret_cast<float4*>(sQ + tk * DS + d + half);
                u = *qu, v = *qv;
                turn4(u, v, c0, c1, 1.0f);
                *qu = u, *qv = v;
            }
        }
    } else {
        for (int i = threadIdx.x; i < cnt * half; i += blockDim.x) {
            const int tk = i / half, m = i % half;
            const int a = tk * DS + (in.interleaved ? 2 * m : m), b = tk * DS + (in.interleaved ? 2 * m + 1 : m + half);
            const float2 c = in.cs[(row + tk) * half + m];
            float u = sK[a], v = sK[b];
            sK[a] = (u * c.x - v * c.y) * f;
            sK[b] = (v * c.x + u * c.y) * f;
            if (sQ) {
                u = sQ[a], v = sQ[b];
                sQ[a] = u * c.x - v * c.y;
                sQ[b] = v * c.x + u * c.y;
            }
        }
    }
    const int rest = D - in.n_rot;
    if (f != 1.0f)
        for (int i = threadIdx.x; i < cnt * rest; i += blockDim.x) sK[(i / rest) * DS + in.n_rot + i % rest] *= f;
}

// Block = up to 128 columns (16 per warp) of one head of one work item. A warp keeps its 16 columns of S transposed in
// accumulators: S[nt][..] = rows (columns of S) g, g + 8 x entries d = 8 nt + 2 t, + 1 (g = lane / 4, t = lane % 4). Summing
// over d may take the entries of a group of eight in any order, so with slot t <-> entry 2 t and slot t + 4 <-> entry 2 t + 1
// the accumulators ARE the B operand of Q S, and Q is read in pairs.
template <int NT>
__global__ void __launch_bounds__(256, 2)
decay_chunk_kernel(DecayIn in, const float* __restrict__ pow_h, int pow_ld, const float* __restrict__ init_buf,
                   float* __restrict__ final_buf, float* __restrict__ o, const int* __restrict__ item_row0,
                   const int* __restrict__ item_n, const int* __restrict__ item_init, const int* __restrict__ item_final,
                   int H, int D, int E, int vec, int vec_v) {
    constexpr int Dp = 8 * NT, DS = Dp + 8;
    extern __shared__ __align__(16) float sm[];
    const int cols = (blockDim.x >> 5) * 16, VS = cols + 8;
    const int stage_floats = kL * (2 * DS + VS);  // two stages of Q | K | V: one is computed on while the other arrives
    float* sA = sm + 2 * stage_floats;
    float* spw = sA + kL * kAS;  // decay^0 .. decay^kL
    const int h = blockIdx.y, b = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
    const int g = lane >> 2, t4 = lane & 3;
    const int e0 = blockIdx.x * cols;
    const int ew = e0 + warp * 16;  // the warp's first column
    const int row0 = item_row0[b], n = item_n[b];
    const int fin = item_final[b];
    if (!o && fin < 0) return;
    const long long de = (long long)D * E;
    for (int i = threadIdx.x; i <= kL; i += blockDim.x) spw[i] = pow_h[(long long)h * pow_ld + i];
    float S[NT][4];
    const float* si = item_init[b] >= 0 ? init_buf + ((long long)item_init[b] * H + h) * de : nullptr;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int d = 8 * nt + 2 * t4 + (c & 1), e = ew + g + (c >> 1) * 8;
            S[nt][c] = (si && d < D && e < E) ? si[(long long)d * E + e] : 0.f;
        }
    auto fetch = [&](int t0, float* base) {
        const int cnt = n - t0 < kL ? n - t0 : kL;
        const float* r = in.src + (row0 + t0) * in.ld;
        if (o) fetch_head(r + in.q_off + (long long)h * D, in.ld, cnt, D, Dp, DS, vec, base);
        fetch_head(r + in.k_off + (long long)h * D, in.ld, cnt, D, Dp, DS, vec, base + kL * DS);
        fetch_head(r + in.v_off + (long long)h * E + e0, in.ld, cnt, E - e0 < cols ? E - e0 : cols, cols, VS, vec_v,
                   base + 2 * kL * DS);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, sm);
    for (int t0 = 0, stage = 0; t0 < n; t0 += kL, stage ^= 1) {
        const int cnt = n - t0 < kL ? n - t0 : kL;
        const long long row = row0 + t0;
        float* sQ = sm + stage * stage_floats;
        float* sK = sQ + kL * DS;
        float* sV = sK + kL * DS;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // this stage is here, and everybody is done with the other one
        if (t0 + kL < n) fetch(t0 + kL, sm + (stage ^ 1) * stage_floats);
        if (in.silu) {
            if (o) silu_rows(sQ, Dp, DS);
            silu_rows(sK, Dp, DS);
            silu_rows(sV, cols, VS);
            if (in.k_scale != 1.0f) turn_rows(in, row, cnt, D, DS, nullptr, sK);
        } else {
            turn_rows(in, row, cnt, D, DS, o ? sQ : nullptr, sK);
        }
        __syncthreads();
        float acc[2][2][4];
        if (o) {
            // A: 16 x 8 tiles on and below the diagonal, a tile per warp at a time
            for (int tile = warp; tile < 6; tile += nwarp) {
                const int mt = tile < 2 ? 0 : 1, nt = tile < 2 ? tile : tile - 2;
                float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f}, c2[4] = {0.f, 0.f, 0.f, 0.f};
                const float* qa = sQ + (mt * 16 + g) * DS + 2 * t4;
                const float* kb = sK + (nt * 8 + g) * DS + 2 * t4;
#pragma unroll
                for (int kk = 0; kk < NT; ++kk) {
                    const float2 x = *reinterpret_cast<const float2*>(qa + 8 * kk);
                    const float2 y = *reinterpret_cast<const float2*>(qa + 8 * DS + 8 * kk);
                    const float2 z = *reinterpret_cast<const float2*>(kb + 8 * kk);
                    FragA a;
                    FragB bb;
                    a.set(x.x, y.x, x.y, y.y);
                    bb.set(z.x, z.y);
                    mma_tf32(c0, a.lo, bb.hi[0], bb.hi[1]);  // three chains: the products of one tile do not wait for one another
                    mma_tf32(c1, a.hi, bb.lo[0], bb.lo[1]);
                    mma_tf32(c2, a.hi, bb.hi[0], bb.hi[1]);
                }
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const int i = mt * 16 + g + (c >> 1) * 8, j = nt * 8 + 2 * t4 + (c & 1);
                    sA[i * kAS + j] = j <= i ? (c0[c] + c1[c] + c2[c]) * spw[i - j] : 0.f;
                }
            }
            // Q S for the warp's columns
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
#pragma unroll
                for (int x = 0; x < 2; ++x)
#pragma unroll
                    for (int c = 0; c < 4; ++c) acc[mt][x][c] = 0.f;
#pragma unroll
            for (int kk = 0; kk < NT; ++kk) {
                FragB b0, b1;
                b0.set(S[kk][0], S[kk][1]);
                b1.set(S[kk][2], S[kk][3]);
#pragma unroll
                for (int mt = 0; mt < 2; ++mt) {
                    const float* qa = sQ + (mt * 16 + g) * DS + 2 * t4 + 8 * kk;
                    const float2 x = *reinterpret_cast<const float2*>(qa);
                    const float2 y = *reinterpret_cast<const float2*>(qa + 8 * DS);
                    FragA a;
                    a.set(x.x, y.x, x.y, y.y);
                    mma3(acc[mt][0], a, b0);
                    mma3(acc[mt][1], a, b1);
                }
            }
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
#pragma unroll
                for (int x = 0; x < 2; ++x)
#pragma unroll
                    for (int c = 0; c < 4; ++c) acc[mt][x][c] *= spw[mt * 16 + g + (c >> 1) * 8 + 1];
            __syncthreads();
            // + A V
#pragma unroll
            for (int ks = 0; ks < kL / 8; ++ks) {
                FragB b0, b1;
                const float* vp = sV + (ks * 8 + t4) * VS + warp * 16 + g;
                b0.set(vp[0], vp[4 * VS]);
                b1.set(vp[8], vp[4 * VS + 8]);
#pragma unroll
                for (int mt = 0; mt < 2; ++mt) {
                    if (mt == 0 && ks >= 2) continue;  // above the diagonal
                    const float* ap = sA + (mt * 16 + g) * kAS + ks * 8 + t4;
                    FragA a;
                    a.set(ap[0], ap[8 * kAS], ap[4], ap[8 * kAS + 4]);
                    mma3(acc[mt][0], a, b0);
                    mma3(acc[mt][1], a, b1);
                }
            }
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
#pragma unroll
                for (int x = 0; x < 2; ++x)
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        const int i = mt * 16 + g + r * 8, e = ew + x * 8 + 2 * t4;
                        if (i >= cnt) continue;
                        float* p = o + (row + i) * H * E + (long long)h * E + e;
                        if (vec_v && e + 1 < E) {
                            *reinterpret_cast<float2*>(p) = make_float2(acc[mt][x][2 * r], acc[mt][x][2 * r + 1]);
                        } else {
                            if (e < E) p[0] = acc[mt][x][2 * r];
                            if (e + 1 < E) p[1] = acc[mt][x][2 * r + 1];
                        }
                    }
        }
        // S <- decay^cnt S + sum_j decay^(cnt - 1 - j) v_j k_j^T (transposed); rows behind cnt are zero in K and V
        const float all = spw[cnt];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int c = 0; c < 4; ++c) S[nt][c] *= all;
#pragma unroll
        for (int ks = 0; ks < kL / 8; ++ks) {
            const int j0 = ks * 8 + t4, j1 = j0 + 4;
            const float w0 = spw[cnt - 1 - j0 > 0 ? cnt - 1 - j0 : 0], w1 = spw[cnt - 1 - j1 > 0 ? cnt - 1 - j1 : 0];
            const float* vp = sV + j0 * VS + warp * 16 + g;
            FragA a;
            a.set(vp[0] * w0, vp[8] * w0, vp[4 * VS] * w1, vp[4 * VS + 8] * w1);
            const float* kp = sK + j0 * DS + g;
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                FragB bb;
                bb.set(kp[8 * nt], kp[4 * DS + 8 * nt]);
                mma3(S[nt], a, bb);
            }
        }
    }
    if (fin < 0) return;
    float* sf = final_buf + ((long long)fin * H + h) * de;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int d = 8 * nt + 2 * t4 + (c & 1), e = ew + g + (c >> 1) * 8;
            if (d < D && e < E) sf[(long long)d * E + e] = S[nt][c];
        }
}

// Between the two chunk passes: on entry chunk_state[w] is what chunk w builds from zero (not read for the last chunk of a
// request), on exit the state it STARTS from: the request's stored state, then S <- decay^(rows of w) S + local_w.
// Up to WB chunks' states are requested before the first is used; V adjacent entries per thread (16-byte accesses with V = 4).
template <int V>
__global__ void decay_combine_kernel(const float* __restrict__ state, float* __restrict__ chunk_state,
                                     const float* __restrict__ pow_h, int pow_ld, const int* __restrict__ item_n,
                                     const int* __restrict__ seq_item0, const int* __restrict__ slot, int H, long long de) {
    constexpr int WB = 8;
    const int h = blockIdx.y, b = blockIdx.z;
    const int w0 = seq_item0[b], w1 = seq_item0[b + 1];
    const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= de) return;
    auto ld = [](const float* p, float (&v)[V]) {
        if constexpr (V == 4) {
            const float4 x = *reinterpret_cast<const float4*>(p);
            v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
        } else {
            v[0] = *p;
        }
    };
    float S[V], loc[WB][V], p[WB];
    ld(state + ((long long)slot[b] * H + h) * de + i, S);
    for (int c0 = w0; c0 < w1; c0 += WB) {
#pragma unroll
        for (int u = 0; u < WB; ++u) {
            p[u] = c0 + u < w1 ? pow_h[(long long)h * pow_ld + item_n[c0 + u]] : 0.f;
            if (c0 + u + 1 < w1) ld(chunk_state + ((long long)(c0 + u) * H + h) * de + i, loc[u]);
        }
#pragma unroll
        for (int u = 0; u < WB; ++u) {
            if (c0 + u >= w1) break;
            float* cs = chunk_state + ((long long)(c0 + u) * H + h) * de + i;
            if constexpr (V == 4) *reinterpret_cast<float4*>(cs) = make_float4(S[0], S[1], S[2], S[3]);
            else *cs = S[0];
            if (c0 + u + 1 < w1) {
#pragma unroll
                for (int v = 0; v < V; ++v) S[v] = fmaf(p[u], S[v], loc[u][v]);
            }
        }
    }
}

static bool bad_in(const float* src, long long ld, const float* cs, int n_rot, int silu, int D) {
    return !src || ld <= 0 || n_rot < 0 || (n_rot % 2) || n_rot > D || (n_rot > 0 && (!cs || silu));
}

}  // namespace decay
}  // namespace llark

using namespace llark;
using namespace llark::decay;

extern "C" int llark_seq_rotary_table(const float* freq, int n_freq, const int* tok_seq, const int* cu, const int* pos0,
                                      float* cs, int n_tok, cudaStream_t st) {
    if (n_freq <= 0 || n_tok <= 0 || !freq || !tok_seq || !cu || !pos0 || !cs) return LLARK_EINVAL;
    const long long n = (long long)n_tok * n_freq;
    const unsigned grid = (unsigned)((n + 255) / 256 < 148 * 8 ? (n + 255) / 256 : 148 * 8);
    rotary_table_kernel<<<grid, 256, 0, st>>>(freq, n_freq, tok_seq, cu, pos0, reinterpret_cast<float2*>(cs), n_tok);
    return check_launch();
}

extern "C" int llark_seq_decay_rows(const float* src, long long ld, int q_off, int k_off, int v_off, const float* cs, int n_rot,
                                    int interleaved, float k_scale, int silu, const float* pow_h, int pow_ld,
                                    const float* init_buf, float* final_buf, float* o, const int* item_row0,
                                    const int* item_n, const int* item_init, const int* item_final, int n_items, int max_n,
                                    int H, int D, int E, cudaStream_t st) {
    if (bad_in(src, ld, cs, n_rot, silu, D) || n_items <= 0 || max_n <= 0 || H <= 0 || D <= 0 || E <= 0 || D > 1024 || !pow_h || pow_ld < 2 ||
        !final_buf || !o || !item_row0 || !item_n || !item_init || !item_final)
        return LLARK_EINVAL;
    const DecayIn in{src, ld, q_off, k_off, v_off, reinterpret_cast<const float2*>(cs), n_rot, interleaved, k_scale, silu};
    int ts = D <= 128 ? 16 : (D <= 512 ? 8 : 4);
    while (ts / 2 >= max_n) ts /= 2;
    const size_t smem = sizeof(float) * (size_t)ts * (2 * D + 32 + 256);
    const int vec = E % 4 == 0 && ((reinterpret_cast<uintptr_t>(init_buf) | reinterpret_cast<uintptr_t>(final_buf)) & 15) == 0;
    const dim3 grid((E + 31) / 32, H, n_items);
#define LLARK_DROWS(RPT)                                                                                                 \
    decay_rows_kernel<RPT><<<grid, 256, smem, st>>>(in, pow_h, pow_ld, init_buf, final_buf, o, item_row0, item_n, item_init, \
                                                    item_final, H, D, E, ts, vec)
    if (D <= 32) LLARK_DROWS(1);
    else if (D <= 64) LLARK_DROWS(2);
    else if (D <= 128) LLARK_DROWS(4);
    else if (D <= 256) LLARK_DROWS(8);
    else if (D <= 512) LLARK_DROWS(16);
    else LLARK_DROWS(32);
#undef LLARK_DROWS
    return check_launch();
}

extern "C" int llark_seq_decay_chunks(const float* src, long long ld, int q_off, int k_off, int v_off, const float* cs,
                                      int n_rot, int interleaved, float k_scale, int silu, const float* pow_h, int pow_ld,
                                      const float* init_buf, float* final_buf, float* o, const int* item_row0,
                                      const int* item_n, const int* item_init, const int* item_final, int n_items, int H,
                                      int D, int E, cudaStream_t st) {
    if (bad_in(src, ld, cs, n_rot, silu, D) || n_items <= 0 || H <= 0 || D <= 0 || E <= 0 || D > 128 || !pow_h || pow_ld < kL + 1 ||
        !final_buf || !item_row0 || !item_n || !item_init || !item_final)
        return LLARK_EINVAL;
    const DecayIn in{src, ld, q_off, k_off, v_off, reinterpret_cast<const float2*>(cs), n_rot, interleaved, k_scale, silu};
    const int warps = E >= 113 ? 8 : (E + 15) / 16;
    const int cols = 16 * warps;
    auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool rows16 = ld % 4 == 0 && al(src);
    if (n_rot && !al(cs)) return LLARK_EINVAL;
    const int vec = rows16 && D % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0;
    const int vec_v = rows16 && E % 4 == 0 && v_off % 4 == 0 && (!o || al(o));
    const dim3 grid((E + cols - 1) / cols, H, n_items);
#define LLARK_DCHUNK(NT)                                                                                                 \
    do {                                                                                                                 \
        const size_t smem = sizeof(float) * (size_t)(2 * kL * (2 * (8 * NT + 8) + cols + 8) + kL * kAS + kL + 4);        \
        if (smem > 48 * 1024) {                                                                                          \
            cudaError_t e = cudaFuncSetAttribute(decay_chunk_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize,     \
                                                 (int)smem);                                                             \
            if (e != cudaSuccess) {                                                                                      \
                g_last_cuda_error = (int)e;                                                                              \
                return LLARK_ECUDA;                                                                                      \
            }                                                                                                            \
        }                                                                                                                \
        decay_chunk_kernel<NT><<<grid, warps * 32, smem, st>>>(in, pow_h, pow_ld, init_buf, final_buf, o, item_row0,      \
                                                               item_n, item_init, item_final, H, D, E, vec, vec_v);       \
    } while (0)
    if (D <= 16) LLARK_DCHUNK(2);
    else if (D <= 32) LLARK_DCHUNK(4);
    else if (D <= 64) LLARK_DCHUNK(8);
    else LLARK_DCHUNK(16);
#undef LLARK_DCHUNK
    return check_launch();
}

extern "C" int llark_seq_decay_combine(const float* state, float* chunk_state, const float* pow_h, int pow_ld,
                                       const int* item_n, const int* seq_item0, const int* slot, int n_seq, int H, int D,
                                       int E, cudaStream_t st) {
    if (n_seq <= 0 || H <= 0 || D <= 0 || E <= 0 || !state || !chunk_state || !pow_h || pow_ld < 2 || !item_n || !seq_item0 ||
        !slot)
        return LLARK_EINVAL;
    const long long de = (long long)D * E;
    const bool vec = de % 4 == 0 && ((reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(chunk_state)) & 15) == 0;
    const dim3 grid((unsigned)((de / (vec ? 4 : 1) + 127) / 128), H, n_seq);
    if (vec)
        decay_combine_kernel<4><<<grid, 128, 0, st>>>(state, chunk_state, pow_h, pow_ld, item_n, seq_item0, slot, H, de);
    else
        decay_combine_kernel<1><<<grid, 128, 0, st>>>(state, chunk_state, pow_h, pow_ld, item_n, seq_item0, slot, H, de);
    return check_launch();
}
