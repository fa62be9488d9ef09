// Routed mixture of experts on the generation path: every token uses `top` of n small feed-forwards
// down(silu(gate x) * (up x)), down(relu(up x)^2) or a clamped gated unit. The router picks experts on the device, one kernel sorts the (token, choice) entries by
// expert and cuts each expert's run into row tiles, and two grouped GEMM launches walk that tile list (rows gathered
// through the sort permutation). Large bf16 steps instead run every expert's rows through the tcgen05 GEMM core in its
// rows-in-runs mode (llark_seq_moe_gather, llark_gemm_segments with the sort kernel's list of 256-row tiles and its
// device-side count, llark_seq_silu_mul). Neither route returns to the host. The
// weighted sum over a token's choices is taken in the order of the choices when the residual is assembled
// (llark_seq_residual_combine), so a token's result does not depend on what else is in the batch.
//
//   llark_seq_moe_route     scores = sigmoid(logits) fp32; experts form `n_groups` groups of neighbours, a group's score
//                           is the sum of its two best, only experts of the best `keep` groups can be chosen; the `top`
//                           best of those; weights = their scores / (sum + 1e-20) * scale
//   llark_seq_moe_route_bias  scores = softmax(logits) fp32 over all router outputs; the CHOICE is made on score +
//                           correction (which may be negative), a group's score is its best choice score, experts outside
//                           the best `keep` groups cannot be chosen; weights = the chosen experts' plain scores * scale,
//                           not renormalised. Router outputs >= n_real are experts without weights that hand their input
//                           through: the sort leaves them out of the tile lists, the residual kernel adds the input.
//   llark_seq_moe_route_top   the `top` largest logits are chosen, weights = softmax over the chosen logits only, or their
//                           sigmoids
//   llark_seq_moe_sort      entries -> perm (sorted by expert), pos_of (inverse), tiles (expert, first row, rows)
//   llark_seq_moe_up        act[pos] = silu(W_gate,e x) * (W_up,e x), or relu(W_up,e x)^2 for experts without a gate;
//                           x = the entry's token row
//   llark_seq_moe_down      z[pos]   = W_down,e act[pos]                 fp32
#include "common.cuh"

namespace llark {
extern thread_local int g_last_cuda_error;
namespace moe {

static int check_launch() {
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) {
        g_last_cuda_error = (int)e;
        return LLARK_ECUDA;
    }
    return LLARK_OK;
}

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float sigmoidf_(float z) { return 1.0f / (1.0f + expf(-z)); }

constexpr int kTileRows = 64;
constexpr int kRowsRouteMaxEntries = 512;  // steps up to this many (token, choice) entries take the weight-streaming kernel

// ------------------------------------------------------------------------------------------------ router
// Warp per token; scores in shared memory. Ties go to the lower expert / group number.
__global__ void route_kernel(const float* __restrict__ logits, long long ld, int* __restrict__ ids,
                             float* __restrict__ wts, int n_tok, int n_exp, int n_groups, int keep, int top,
                             float scale) {
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const long long t = (long long)blockIdx.x * nw + warp;
    if (t >= n_tok) return;
    float* s = sm + (long long)warp * (n_exp + n_groups);   // scores; -1 once taken or shut out
    float* gs = s + n_exp;                                  // group scores
    const int per = n_exp / n_groups;
    for (int e = lane; e < n_exp; e += 32) s[e] = sigmoidf_(logits[t * ld + e]);
    __syncwarp();
    for (int g = lane; g < n_groups; g += 32) {
        float a = -1.f, b = -1.f;  // the two largest (scores are positive)
        for (int i = 0; i < per; ++i) {
            const float v = s[g * per + i];
            if (v > a) {
                b = a;
                a = v;
            } else if (v > b) {
                b = v;
            }
        }
        gs[g] = a + (b > 0.f ? b : 0.f);
    }
    __syncwarp();
    if (keep < n_groups) {
        if (lane == 0) {
            for (int r = 0; r < keep; ++r) {  // mark the best `keep` groups with a negative score - 2 (still ordered)
                int best = -1;
                float bv = -1.f;
                for (int g = 0; g < n_groups; ++g)
                    if (gs[g] >= 0.f && gs[g] > bv) {
                        bv = gs[g];
                        best = g;
                    }
                gs[best] = -2.f;
            }
        }
        __syncwarp();
        for (int e = lane; e < n_exp; e += 32)
            if (gs[e / per] != -2.f) s[e] = -1.f;
        __syncwarp();
    }
    float chosen_w = 0.f;  // lane k keeps choice k (top <= 32)
    int chosen_e = 0;
    float sum = 0.f;
    for (int k = 0; k < top; ++k) {
        float bv = -1.f;
        int be = 0x7fffffff;
        for (int e = lane; e < n_exp; e += 32)
            if (s[e] > bv) {
                bv = s[e];
                be = e;
            }
        for (int m = 16; m > 0; m >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, m);
            const int oe = __shfl_xor_sync(0xffffffffu, be, m);
            if (ov > bv || (ov == bv && oe < be)) {
                bv = ov;
                be = oe;
            }
        }
        if (lane == k) {
            chosen_w = bv;
            chosen_e = be;
        }
        sum += bv;
        if (lane == 0) s[be] = -1.f;
        __syncwarp();
    }
    if (lane < top) {
        ids[t * top + lane] = chosen_e;
        wts[t * top + lane] = chosen_w / (sum + 1e-20f) * scale;
    }
}

// Warp per token. s = plain scores, c = choice scores (-inf once taken or shut out). Ties go to the lower number.
__global__ void route_bias_kernel(const float* __restrict__ logits, long long ld, const float* __restrict__ correction,
                                  int* __restrict__ ids, float* __restrict__ wts, int n_tok, int n_exp, int n_groups,
                                  int keep, int top, float scale) {
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const long long t = (long long)blockIdx.x * nw + warp;
    if (t >= n_tok) return;
    float* s = sm + (long long)warp * (2 * n_exp + n_groups);
    float* c = s + n_exp;
    float* gs = c + n_exp;
    const int per = n_exp / n_groups;
    float mx = -INFINITY;
    for (int e = lane; e < n_exp; e += 32) mx = fmaxf(mx, logits[t * ld + e]);
    mx = warp_max(mx);
    float den = 0.f;
    for (int e = lane; e < n_exp; e += 32) {
        const float v = expf(logits[t * ld + e] - mx);
        s[e] = v;
        den += v;
    }
    den = warp_sum(den);
    for (int e = lane; e < n_exp; e += 32) {
        s[e] = s[e] / den;
        c[e] = s[e] + (correction ? correction[e] : 0.f);
    }
    __syncwarp();
    if (keep < n_groups) {
        for (int g = lane; g < n_groups; g += 32) {
            float a = -INFINITY;
            for (int i = 0; i < per; ++i) a = fmaxf(a, c[g * per + i]);
            gs[g] = a;
        }
        __syncwarp();
        if (lane == 0) {
            for (int r = 0; r < keep; ++r) {  // the best `keep` groups are marked with +inf
                int best = -1;
                float bv = -INFINITY;
                for (int g = 0; g < n_groups; ++g)
                    if (gs[g] != INFINITY && (best < 0 || gs[g] > bv)) {
                        bv = gs[g];
                        best = g;
                    }
                gs[best] = INFINITY;
            }
        }
        __syncwarp();
        for (int e = lane; e < n_exp; e += 32)
            if (gs[e / per] != INFINITY) c[e] = -INFINITY;
        __syncwarp();
    }
    float chosen_w = 0.f;  // lane k keeps choice k (top <= 32)
    int chosen_e = 0;
    for (int k = 0; k < top; ++k) {
        float bv = -INFINITY;
        int be = 0x7fffffff;
        for (int e = lane; e < n_exp; e += 32)
            if (c[e] > bv) {
                bv = c[e];
                be = e;
            }
        for (int m = 16; m > 0; m >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, m);
            const int oe = __shfl_xor_sync(0xffffffffu, be, m);
            if (ov > bv || (ov == bv && oe < be)) {
                bv = ov;
                be = oe;
            }
        }
        if (lane == k) {
            chosen_e = be;
            chosen_w = s[be];
        }
        __syncwarp();
        if (lane == 0) c[be] = -INFINITY;
        __syncwarp();
    }
    if (lane < top) {
        ids[t * top + lane] = chosen_e;
        wts[t * top + lane] = chosen_w * scale;
    }
}

// Warp per token, logits in shared memory. The choice is made on the logits themselves (a softmax over all of them could
// underflow, a sigmoid saturate, and lose the order); ties go to the lower number. Weights: softmax over the chosen logits,
// or, sigmoid_wts, the sigmoid of each as it is.
__global__ void route_top_kernel(const float* __restrict__ logits, long long ld, int* __restrict__ ids,
                                 float* __restrict__ wts, int n_tok, int n_exp, int top, int sigmoid_wts) {
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const long long t = (long long)blockIdx.x * nw + warp;
    if (t >= n_tok) return;
    float* s = sm + (long long)warp * n_exp;  // logits; -inf once taken
    for (int e = lane; e < n_exp; e += 32) s[e] = logits[t * ld + e];
    __syncwarp();
    float chosen = -INFINITY, first = 0.f;  // lane k keeps choice k (top <= 32)
    int chosen_e = 0;
    for (int k = 0; k < top; ++k) {
        float bv = -INFINITY;
        int be = 0x7fffffff;
        for (int e = lane; e < n_exp; e += 32)
            if (s[e] > bv) {
                bv = s[e];
                be = e;
            }
        for (int m = 16; m > 0; m >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, m);
            const int oe = __shfl_xor_sync(0xffffffffu, be, m);
            if (ov > bv || (ov == bv && oe < be)) {
                bv = ov;
                be = oe;
            }
        }
        if (be >= n_exp) be = 0;  // no number compared greater (NaN logits): stay inside the tables
        if (k == 0) first = bv;
        if (lane == k) {
            chosen = bv;
            chosen_e = be;
        }
        if (lane == 0) s[be] = -INFINITY;
        __syncwarp();
    }
    const float w = lane < top ? expf(chosen - first) : 0.f;
    const float sum = warp_sum(w);
    if (lane < top) {
        ids[t * top + lane] = chosen_e;
        wts[t * top + lane] = sigmoid_wts ? sigmoidf_(chosen) : w / sum;
    }
}

// ------------------------------------------------------------------------------------------------ sort by expert
// One block. meta[0] = number of tiles; tiles[i] = (expert, first sorted row, rows). Experts >= n_real (no weights) keep
// their place in the sorted order but get no tiles.
__global__ void sort_kernel(const int* __restrict__ ids, int n_ent, int n_exp, int n_real, int* __restrict__ perm,
                            int* __restrict__ pos_of, int* __restrict__ tiles, int* __restrict__ meta,
                            int* __restrict__ seg_off, int* __restrict__ tiles256) {
    extern __shared__ int si[];
    int* cnt = si;               // [n_exp]
    int* off = cnt + n_exp;      // [n_exp + 1]
    int* cur = off + n_exp + 1;  // [n_exp]
    for (int e = threadIdx.x; e < n_exp; e += blockDim.x) cnt[e] = cur[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n_ent; i += blockDim.x) atomicAdd(&cnt[ids[i]], 1);
    __syncthreads();
    if (threadIdx.x == 32 && tiles256) {  // the GEMM core's tile list (256-row m-blocks), by another warp
        int o = 0, nt = 0;
        for (int e = 0; e < n_real; ++e) {
            for (int r = 0; r < cnt[e]; r += 256) {
                tiles256[3 * nt] = e;
                tiles256[3 * nt + 1] = o + r;
                tiles256[3 * nt + 2] = cnt[e] - r < 256 ? cnt[e] - r : 256;
                ++nt;
            }
            o += cnt[e];
        }
        meta[1] = nt;
    }
    if (threadIdx.x == 0) {
        int o = 0, nt = 0;
        for (int e = 0; e < n_exp; ++e) {
            off[e] = o;
            for (int r = 0; e < n_real && r < cnt[e]; r += kTileRows) {
                tiles[3 * nt] = e;
                tiles[3 * nt + 1] = o + r;
                tiles[3 * nt + 2] = cnt[e] - r < kTileRows ? cnt[e] - r : kTileRows;
                ++nt;
            }
            o += cnt[e];
        }
        off[n_exp] = o;
        meta[0] = nt;
    }
    __syncthreads();
    if (seg_off)
        for (int e = threadIdx.x; e <= n_exp; e += blockDim.x) seg_off[e] = off[e];
    for (int i = threadIdx.x; i < n_ent; i += blockDim.x) {
        const int e = ids[i];
        const int p = off[e] + atomicAdd(&cur[e], 1);
        perm[p] = i;
        pos_of[i] = p;
    }
}

// ------------------------------------------------------------------------------------------------ grouped GEMMs
// Block = one row tile of one expert x 64 output columns. MODE kSiluGlu: two weight matrices (gate rows, then up rows, of the
// expert's [2 * N, K] block) and out = silu(a) * b; kRelu2: out = relu(product)^2; kPlain: the product. Rows of A:
// gather ? perm[pos] / top : pos.
// kClampGlu: gate and up rows of the expert's [2 * N, K] block alternate, out = g' * sigmoid(slope g') * (u' + 1) with
// g' = min(g, limit), u' = clamp(u, -limit, limit). in_wts (optional): entry i = perm[pos] of the step is multiplied by
// in_wts[i] on its way in, which is done on the sums (W (c x) = c (W x)).
enum { kPlain = 0, kSiluGlu = 1, kRelu2 = 2, kClampGlu = 3 };

struct UpArgs {
    const float* in_wts;
    float limit, slope;
};
__device__ __forceinline__ float clamp_glu(const UpArgs& a, float g, float u) {
    g = fminf(g, a.limit);
    return g / (1.0f + expf(-a.slope * g)) * (fminf(fmaxf(u, -a.limit), a.limit) + 1.0f);
}

template <typename T, typename TC, int MODE>
__global__ void __launch_bounds__(256)
grouped_linear_kernel(const T* __restrict__ A, long long lda, const int* __restrict__ perm, int top,
                      const T* __restrict__ W, TC* __restrict__ Cm, long long ldc, const int* __restrict__ tiles,
                      const int* __restrict__ meta, int N, int K, UpArgs up) {
    constexpr int BM = kTileRows, BN = 64, BK = 16;
    constexpr bool DUAL = MODE == kSiluGlu || MODE == kClampGlu;
    constexpr int STEP = MODE == kClampGlu ? 2 : 1;  // weight rows from one gate (up) row to the next
    const int up0 = MODE == kClampGlu ? 1 : N;       // the first up row
    if ((int)blockIdx.y >= meta[0]) return;
    __shared__ float As[BK][BM + 4];
    __shared__ float Ws[DUAL ? 2 : 1][BK][BN + 4];
    __shared__ int rows[BM];
    const int ex = tiles[3 * blockIdx.y], r0 = tiles[3 * blockIdx.y + 1], nr = tiles[3 * blockIdx.y + 2];
    const T* We = W + (long long)ex * (DUAL ? 2 : 1) * N * K;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int n0 = blockIdx.x * BN;
    for (int i = threadIdx.x; i < BM; i += 256) rows[i] = i < nr ? (perm ? perm[r0 + i] / top : r0 + i) : -1;
    __syncthreads();
    float acc[4][4] = {}, acc2[DUAL ? 4 : 1][4] = {};
    for (int k0 = 0; k0 < K; k0 += BK) {
        for (int i = threadIdx.x; i < BM * BK; i += 256) {
            const int r = i / BK, k = i % BK;
            As[k][r] = (rows[r] >= 0 && k0 + k < K) ? ldf(A + (long long)rows[r] * lda + k0 + k) : 0.f;
            const bool in = n0 + r < N && k0 + k < K;
            Ws[0][k][r] = in ? ldf(We + (long long)(n0 + r) * STEP * K + k0 + k) : 0.f;
            if (DUAL) Ws[1][k][r] = in ? ldf(We + ((long long)(n0 + r) * STEP + up0) * K + k0 + k) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; ++k) {
            float a[4], b[4], b2[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = As[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                b[j] = Ws[0][k][tx * 4 + j];
                if (DUAL) b2[j] = Ws[1][k][tx * 4 + j];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
                    if (DUAL) acc2[i][j] = fmaf(a[i], b2[j], acc2[i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int m = ty * 4 + i, n = n0 + tx * 4 + j;
            if (m < nr && n < N) {
                float y = acc[i][j];
                const float c = up.in_wts ? up.in_wts[perm[r0 + m]] : 1.0f;
                y *= c;
                if (MODE == kSiluGlu) y = y * sigmoidf_(y) * (c * acc2[i][j]);
                if (MODE == kClampGlu) y = clamp_glu(up, y, c * acc2[i][j]);
                if (MODE == kRelu2) {
                    y = fmaxf(y, 0.f);
                    y *= y;
                }
                stf(Cm + (long long)(r0 + m) * ldc + n, y);
            }
        }
}

// Few rows per expert (decode): a warp owns one output column of one row tile (gated units: its gate and its up row) or two
// adjacent ones (kPlain, kRelu2) and streams the two weight rows in 16-byte pieces; the tile's rows come from L1 / L2, MB at a
// time, and are read once for both. A small MB keeps the registers few and the warps many, which pays as long as an expert
// has a handful of rows (the second pass over a weight row comes from L1).
template <typename T, typename TC, int MODE, int MB>
__global__ void __launch_bounds__(256)
grouped_rows_kernel(const T* __restrict__ A, long long lda, const int* __restrict__ perm, int top,
                    const T* __restrict__ W, TC* __restrict__ Cm, long long ldc, const int* __restrict__ tiles,
                    const int* __restrict__ meta, int N, int K, int vec_ok, UpArgs up) {
    constexpr int VEC = 16 / (int)sizeof(T);
    constexpr bool DUAL = MODE == kSiluGlu || MODE == kClampGlu;
    if ((int)blockIdx.y >= meta[0]) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n = (blockIdx.x * (blockDim.x >> 5) + warp) * (DUAL ? 1 : 2);
    if (n >= N) return;
    const int ex = tiles[3 * blockIdx.y], r0 = tiles[3 * blockIdx.y + 1], nr = tiles[3 * blockIdx.y + 2];
    const T* w1 = W + ((long long)ex * (DUAL ? 2 : 1) * N + (MODE == kClampGlu ? 2 * n : n)) * K;
    const T* w2 = w1 + (MODE == kSiluGlu ? (long long)N * K
                                         : (MODE == kClampGlu || n + 1 < N ? (long long)K : 0));  // tail: re-read, never stored
    for (int m0 = 0; m0 < nr; m0 += MB) {
        const T* ar[MB];
#pragma unroll
        for (int m = 0; m < MB; ++m) {
            const int p = r0 + (m0 + m < nr ? m0 + m : nr - 1);
            ar[m] = A + (long long)(perm ? perm[p] / top : p) * lda;
        }
        float acc[MB], acc2[MB];
#pragma unroll
        for (int m = 0; m < MB; ++m) acc[m] = acc2[m] = 0.f;
        int k0 = 0;
        if (vec_ok) {
            const int kv = K / VEC;
            for (int v = lane; v < kv; v += 32) {
                const uint4 wa = __ldcs(reinterpret_cast<const uint4*>(w1) + v);
                const uint4 wb = __ldcs(reinterpret_cast<const uint4*>(w2) + v);
                const T* pa = reinterpret_cast<const T*>(&wa);
                const T* pb = reinterpret_cast<const T*>(&wb);
#pragma unroll
                for (int m = 0; m < MB; ++m) {
                    if (m0 + m < nr) {
                        const uint4 av = __ldg(reinterpret_cast<const uint4*>(ar[m]) + v);
                        const T* px = reinterpret_cast<const T*>(&av);
#pragma unroll
                        for (int e = 0; e < VEC; ++e) {
                            const float xv = ldf(px + e);
                            acc[m] = fmaf(xv, ldf(pa + e), acc[m]);
                            acc2[m] = fmaf(xv, ldf(pb + e), acc2[m]);
                        }
                    }
                }
            }
            k0 = kv * VEC;
        }
        for (int k = k0 + lane; k < K; k += 32) {
            const float wa = ldf(w1 + k), wb = ldf(w2 + k);
#pragma unroll
            for (int m = 0; m < MB; ++m)
                if (m0 + m < nr) {
                    const float xv = ldf(ar[m] + k);
                    acc[m] = fmaf(xv, wa, acc[m]);
                    acc2[m] = fmaf(xv, wb, acc2[m]);
                }
        }
#pragma unroll
        for (int m = 0; m < MB; ++m) {
            float y = warp_sum(acc[m]), u = warp_sum(acc2[m]);
            if (up.in_wts && m0 + m < nr) {
                const float c = up.in_wts[perm[r0 + m0 + m]];
                y *= c, u *= c;
            }
            if (MODE == kSiluGlu) y = y * sigmoidf_(y) * u;
            if (MODE == kClampGlu) y = clamp_glu(up, y, u);
            if (MODE == kRelu2) {
                y = fmaxf(y, 0.f), u = fmaxf(u, 0.f);
                y *= y, u *= u;
            }
            if (lane == 0 && m0 + m < nr) {
                TC* c = Cm + (long long)(r0 + m0 + m) * ldc + n;
                stf(c, y);
                if (!DUAL && n + 1 < N) stf(c + 1, u);
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ dense-GEMM route
// Large steps run each expert's rows through the framework's GEMM core instead: rows gathered into sorted order first (each
// multiplied by its weight where the unit wants it so), silu(gate) * up afterwards.
template <typename T>
__global__ void gather_rows_kernel(const T* __restrict__ x, long long ldx, const int* __restrict__ perm, int top,
                                   T* __restrict__ xs, int C, const float* __restrict__ in_wts) {
    const long long p = blockIdx.x;
    const T* src = x + (long long)(perm[p] / top) * ldx;
    T* dst = xs + p * C;
    const float c = in_wts ? in_wts[perm[p]] : 1.0f;
    if ((C * (int)sizeof(T)) % 16 == 0 && (ldx * (long long)sizeof(T)) % 16 == 0) {
        constexpr int VEC = 16 / (int)sizeof(T);
        const int nv = C / VEC;
        for (int i = threadIdx.x; i < nv; i += blockDim.x) {
            uint4 v = reinterpret_cast<const uint4*>(src)[i];
            if (in_wts) {
                T* e = reinterpret_cast<T*>(&v);
#pragma unroll
                for (int j = 0; j < VEC; ++j) stf(e + j, c * ldf(e + j));
            }
            reinterpret_cast<uint4*>(dst)[i] = v;
        }
    } else {
        for (int i = threadIdx.x; i < C; i += blockDim.x) stf(dst + i, c * ldf(src + i));
    }
}

template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gu, T* __restrict__ act, long long rows, int ff) {
    const long long n = rows * ff;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / ff;
        const int c = (int)(i % ff);
        const float g = ldf(gu + r * 2 * ff + c), u = ldf(gu + r * 2 * ff + ff + c);
        stf(act + i, g * sigmoidf_(g) * u);
    }
}

}  // namespace moe
}  // namespace llark

using namespace llark;
using namespace llark::moe;
typedef __nv_bfloat16 bf16_t;

extern "C" int llark_seq_moe_route(const float* logits, long long ld, int* ids, float* wts, int n_tok, int n_exp,
                                   int n_groups, int keep, int top, float scale, cudaStream_t st) {
    if (n_tok <= 0 || n_exp <= 0 || n_groups <= 0 || (n_exp % n_groups) || keep <= 0 || keep > n_groups || top <= 0 ||
        top > 32 || top > keep * (n_exp / n_groups) || !logits || !ids || !wts)
        return LLARK_EINVAL;
    const int nw = 4;
    const size_t smem = sizeof(float) * nw * (size_t)(n_exp + n_groups);
    if (smem > 48 * 1024) return LLARK_EINVAL;
    route_kernel<<<(n_tok + nw - 1) / nw, nw * 32, smem, st>>>(logits, ld, ids, wts, n_tok, n_exp, n_groups, keep, top,
                                                              scale);
    return check_launch();
}

extern "C" int llark_seq_moe_route_bias(const float* logits, long long ld, const float* correction, int* ids, float* wts,
                                        int n_tok, int n_exp, int n_groups, int keep, int top, float scale,
                                        cudaStream_t st) {
    if (n_tok <= 0 || n_exp <= 0 || n_groups <= 0 || (n_exp % n_groups) || keep <= 0 || keep > n_groups || top <= 0 ||
        top > 32 || top > keep * (n_exp / n_groups) || !logits || !ids || !wts)
        return LLARK_EINVAL;
    const int nw = 4;
    const size_t smem = sizeof(float) * nw * (size_t)(2 * n_exp + n_groups);
    if (smem > 48 * 1024) return LLARK_EINVAL;
    route_bias_kernel<<<(n_tok + nw - 1) / nw, nw * 32, smem, st>>>(logits, ld, correction, ids, wts, n_tok, n_exp,
                                                                   n_groups, keep, top, scale);
    return check_launch();
}

extern "C" int llark_seq_moe_route_top(const float* logits, long long ld, int* ids, float* wts, int n_tok, int n_exp, int top,
                                       int sigmoid_wts, cudaStream_t st) {
    if (n_tok <= 0 || n_exp <= 0 || top <= 0 || top > 32 || top > n_exp || !logits || !ids || !wts) return LLARK_EINVAL;
    const int nw = 4;
    const size_t smem = sizeof(float) * nw * (size_t)n_exp;
    if (smem > 48 * 1024) return LLARK_EINVAL;
    route_top_kernel<<<(n_tok + nw - 1) / nw, nw * 32, smem, st>>>(logits, ld, ids, wts, n_tok, n_exp, top, sigmoid_wts);
    return check_launch();
}

extern "C" int llark_seq_moe_tile_rows(void) { return kTileRows; }

extern "C" int llark_seq_moe_sort(const int* ids, int n_ent, int n_exp, int n_real, int* perm, int* pos_of, int* tiles,
                                  int* meta, int* seg_off, int* tiles256, cudaStream_t st) {
    if (n_ent <= 0 || n_exp <= 0 || n_real < 0 || n_real > n_exp || !ids || !perm || !pos_of || !tiles || !meta)
        return LLARK_EINVAL;
    const size_t smem = sizeof(int) * (3 * (size_t)n_exp + 1);
    if (smem > 48 * 1024) return LLARK_EINVAL;
    sort_kernel<<<1, 1024, smem, st>>>(ids, n_ent, n_exp, n_real, perm, pos_of, tiles, meta, seg_off, tiles256);
    return check_launch();
}

template <typename T, typename TC, int MODE>
static void launch_rows(const T* A, long long lda, const int* perm, int top, const T* W, TC* C, const int* tiles,
                        const int* meta, int max_tiles, int n_ent, int N, int K, int vec_ok, UpArgs up, cudaStream_t st) {
    const int per = MODE == kSiluGlu || MODE == kClampGlu ? 8 : 16;  // output columns of a block's eight warps
    const dim3 grid((N + per - 1) / per, max_tiles);
    const int n_exp = max_tiles - (n_ent + kTileRows - 1) / kTileRows;
    if (n_ent <= 8 * n_exp)  // a handful of rows per expert
        grouped_rows_kernel<T, TC, MODE, 2><<<grid, 256, 0, st>>>(A, lda, perm, top, W, C, N, tiles, meta, N, K, vec_ok, up);
    else
        grouped_rows_kernel<T, TC, MODE, 8><<<grid, 256, 0, st>>>(A, lda, perm, top, W, C, N, tiles, meta, N, K, vec_ok, up);
}

template <typename T, int MODE>
static int launch_up(const void* x, long long ldx, const int* perm, int top, const void* w, void* act, const int* tiles,
                     const int* meta, int max_tiles, int n_ent, int ff, int K, UpArgs up, cudaStream_t st) {
    if (n_ent <= kRowsRouteMaxEntries) {  // a handful of rows per expert: stream the weights once
        const int vec = 16 / (int)sizeof(T);
        const int vec_ok = (K % vec == 0) && (ldx % vec == 0) &&
                           (((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15) == 0);
        launch_rows<T, T, MODE>((const T*)x, ldx, perm, top, (const T*)w, (T*)act, tiles, meta, max_tiles, n_ent, ff, K,
                                vec_ok, up, st);
    } else {
        grouped_linear_kernel<T, T, MODE><<<dim3((ff + 63) / 64, max_tiles), 256, 0, st>>>(
            (const T*)x, ldx, perm, top, (const T*)w, (T*)act, ff, tiles, meta, ff, K, up);
    }
    return check_launch();
}

// gated = 1: w holds gate rows, then up rows, [n, 2 * ff, K], act = silu(gate x) * (up x); gated = 0: w is [n, ff, K],
// act = relu(w x)^2; gated = 2: gate and up rows alternate, the clamped gated unit with `limit` and `slope`
extern "C" int llark_seq_moe_up(const void* x, long long ldx, const int* perm, int top, const void* w, void* act,
                                const int* tiles, const int* meta, int max_tiles, int n_ent, int ff, int K, int gated,
                                const float* in_wts, float limit, float slope, int act_fp32, cudaStream_t st) {
    if (max_tiles <= 0 || ff <= 0 || K <= 0 || top <= 0 || gated < 0 || gated > 2 || !x || !perm || !w || !act || !tiles || !meta)
        return LLARK_EINVAL;
    const UpArgs up{in_wts, limit, slope};
#define LLARK_UP(T, MODE) launch_up<T, MODE>(x, ldx, perm, top, w, act, tiles, meta, max_tiles, n_ent, ff, K, up, st)
    if (gated == 2) return act_fp32 ? LLARK_UP(float, kClampGlu) : LLARK_UP(bf16_t, kClampGlu);
    if (gated == 1) return act_fp32 ? LLARK_UP(float, kSiluGlu) : LLARK_UP(bf16_t, kSiluGlu);
    return act_fp32 ? LLARK_UP(float, kRelu2) : LLARK_UP(bf16_t, kRelu2);
#undef LLARK_UP
}

extern "C" int llark_seq_moe_down(const void* act, const void* w_down, float* z, const int* tiles, const int* meta,
                                  int max_tiles, int n_ent, int C, int ff, int act_fp32, cudaStream_t st) {
    if (max_tiles <= 0 || ff <= 0 || C <= 0 || !act || !w_down || !z || !tiles || !meta) return LLARK_EINVAL;
    if (n_ent <= kRowsRouteMaxEntries) {
        const int esz = act_fp32 ? 4 : 2, vec = 16 / esz;
        const int vec_ok = (ff % vec == 0) &&
                           (((reinterpret_cast<uintptr_t>(act) | reinterpret_cast<uintptr_t>(w_down)) & 15) == 0);
        if (act_fp32)
            launch_rows<float, float, kPlain>((const float*)act, ff, nullptr, 1, (const float*)w_down, z, tiles, meta,
                                              max_tiles, n_ent, C, ff, vec_ok, UpArgs{}, st);
        else
            launch_rows<bf16_t, float, kPlain>((const bf16_t*)act, ff, nullptr, 1, (const bf16_t*)w_down, z, tiles, meta,
                                               max_tiles, n_ent, C, ff, vec_ok, UpArgs{}, st);
        return check_launch();
    }
    dim3 grid((C + 63) / 64, max_tiles);
    if (act_fp32)
        grouped_linear_kernel<float, float, kPlain><<<grid, 256, 0, st>>>((const float*)act, ff, nullptr, 1,
                                                                         (const float*)w_down, z, C, tiles, meta, C, ff, UpArgs{});
    else
        grouped_linear_kernel<bf16_t, float, kPlain><<<grid, 256, 0, st>>>((const bf16_t*)act, ff, nullptr, 1,
                                                                          (const bf16_t*)w_down, z, C, tiles, meta, C, ff, UpArgs{});
    return check_launch();
}

extern "C" int llark_seq_moe_gather(const void* x, long long ldx, const int* perm, int top, void* xs, int n_ent, int C,
                                    const float* in_wts, int act_fp32, cudaStream_t st) {
    if (n_ent <= 0 || C <= 0 || top <= 0 || !x || !perm || !xs) return LLARK_EINVAL;
    if (act_fp32)
        gather_rows_kernel<float><<<n_ent, 128, 0, st>>>((const float*)x, ldx, perm, top, (float*)xs, C, in_wts);
    else
        gather_rows_kernel<bf16_t><<<n_ent, 128, 0, st>>>((const bf16_t*)x, ldx, perm, top, (bf16_t*)xs, C, in_wts);
    return check_launch();
}

extern "C" int llark_seq_silu_mul(const void* gu, void* act, long long rows, int ff, int act_fp32, cudaStream_t st) {
    if (rows <= 0 || ff <= 0 || !gu || !act) return LLARK_EINVAL;
    const long long n = rows * ff;
    const unsigned grid = (unsigned)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
    if (act_fp32)
        silu_mul_kernel<float><<<grid, 256, 0, st>>>((const float*)gu, (float*)act, rows, ff);
    else
        silu_mul_kernel<bf16_t><<<grid, 256, 0, st>>>((const bf16_t*)gu, (bf16_t*)act, rows, ff);
    return check_launch();
}
