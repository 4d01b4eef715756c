// A decayed sum of outer products with one fixed decay per head (linear attention of the retention and lightning kind):
//
//     S_t = decay_h * S_{t-1} + k_t v_t^T;      o_t = q_scale * S_t^T q_t
//
// per head, S [rows, cols] (key size x value size) float in the request's state slot, column by column ([heads, cols,
// rows]).  q, k and v may pass SiLU on their way in (`act`).  Memory is never cleared: a sequence whose first token of
// the step sits at position 0 starts from zeros whatever its slot holds.  `powers` [heads, FD_C + 1] holds decay^0 ..
// decay^FD_C of every head (entry 1 is the decay itself).
//
// Two ways of computing the same sum:
//
//  * The walk (float and bfloat16, any sizes): token by token, the state in registers, no shared memory and no barrier.
//    A column of S is shared by LPC neighbouring lanes (RPL rows each, one run of floats), a lane group owns NC
//    neighbouring columns.  The NC sums over the rows of a token are taken together: lanes exchange halves of what they
//    hold, so that NC sums over 32 lanes cost 9 shuffles instead of 5 NC.  The next tokens' vectors are in flight
//    while the current ones are used.  This is the decode step, and the float32 path.
//
//  * Chunks of FD_C tokens (bfloat16, sequences that bring many tokens), because the decay does not depend on the data:
//    with i, j counted inside a chunk of L tokens and S the state before it,
//        o_i = q_scale * ( decay^{i+1} S^T q_i  +  sum_{j <= i} decay^{i-j} (q_i . k_j) v_j )
//        S'  = decay^L S + sum_j decay^{L-1-j} k_j v_j^T
//    A first kernel walks the chunks of a (sequence, head): the state stays float, in the accumulators of its matrix
//    products, and what it was before every chunk is left in scratch memory.  A second kernel does all chunks at once.
//    Everything is mma.sync with bfloat16 operands and float accumulators; what is not bfloat16 to begin with (the
//    state, the decayed keys, the decayed scores) enters a product as the sum of two bfloat16 numbers (16 bits of
//    mantissa), so that the chunked form has the inputs' rounding and the outputs' and no other of that size.
//    The scratch holds the state in the order in which the second kernel's lanes want their operand registers:
//    a lane stores and loads 16 bytes (both halves of both words) and neither kernel turns anything round.
//
// Every sequence of a step takes the walk or the chunks by its own number of tokens alone.
#include "common.cuh"
#include "attention_mma.cuh"       // ldmatrix_x4, ldmatrix_x4_trans, mma_bf16_16816, pack_bf16

using namespace vapi;

constexpr int FD_C = 128;          // tokens of a chunk
constexpr int FD_THREADS = 128;

__device__ __forceinline__ float fd_silu(float z) { return z / (1.f + expf(-z)); }
// the same where the result is rounded to 16 bits or split into two such halves
__device__ __forceinline__ float fd_silu_16(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// ---- the walk -------------------------------------------------------------------------------------------
template <typename T> struct FdRaw4;                                  // four elements as they lie in memory
template <> struct FdRaw4<float> {
    float4 x;
    __device__ __forceinline__ float4 f32() const { return x; }
};
template <> struct FdRaw4<__nv_bfloat16> {
    uint2 x;
    __device__ __forceinline__ float4 f32() const {
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
};
__device__ __forceinline__ FdRaw4<float> fd_pack4(float a, float b, float c, float d, float) {
    FdRaw4<float> r; r.x = make_float4(a, b, c, d); return r;
}
__device__ __forceinline__ FdRaw4<__nv_bfloat16> fd_pack4(__nv_bfloat16 a, __nv_bfloat16 b, __nv_bfloat16 c, __nv_bfloat16 d, __nv_bfloat16) {
    FdRaw4<__nv_bfloat16> r;
    __nv_bfloat162 lo = __halves2bfloat162(a, b), hi = __halves2bfloat162(c, d);
    r.x.x = *reinterpret_cast<unsigned*>(&lo);
    r.x.y = *reinterpret_cast<unsigned*>(&hi);
    return r;
}
// elements p[0 .. 3] of which the first `left` exist (the others read as zero)
template <typename T>
__device__ __forceinline__ FdRaw4<T> fd_load4(const T* p, int left, bool wide) {
    const T z = from_f32<T>(0.f);
    if (left <= 0) return fd_pack4(z, z, z, z, z);
    if (wide) return *reinterpret_cast<const FdRaw4<T>*>(p);           // (sizes come in fours then)
    return fd_pack4(p[0], left > 1 ? p[1] : z, left > 2 ? p[2] : z, left > 3 ? p[3] : z, z);
}
__device__ __forceinline__ float4 fd_act4(float4 v, int act) {
    if (act) { v.x = fd_silu(v.x); v.y = fd_silu(v.y); v.z = fd_silu(v.z); v.w = fd_silu(v.w); }
    return v;
}

// TG: tokens in flight (one in decode steps: fewer registers, more warps with their part of a state under way)
template <typename T, int RPL, int LPC, int NC, int TG>
__global__ void __launch_bounds__(FD_THREADS)
fixed_decay_walk_kernel(const T* __restrict__ qkv, long long qkv_stride, int q_off, int k_off, int v_off,
                        const float* __restrict__ powers, float q_scale, int act, float* __restrict__ state, long long slot_stride,
                        const int* __restrict__ state_slots, const int* __restrict__ cu_q, const int* __restrict__ positions,
                        float* __restrict__ out, int nh, int rows, int cols, int num_slots, int q_below, int wide,
                        int* __restrict__ status) {
    static_assert(RPL % 4 == 0 && NC % 4 == 0 && NC <= LPC, "rows and columns of a lane come in fours");
    constexpr int GROUPS = 32 / LPC;
    const int s = blockIdx.z, h = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int grp = lane / LPC, sl = lane % LPC;
    const int col0 = ((blockIdx.x * (FD_THREADS / 32) + warp) * GROUPS + grp) * NC;      // this lane group's columns
    const int r0 = sl * RPL;
    const int t0 = cu_q[s], qlen = cu_q[s + 1] - t0;
    if (qlen <= 0 || (q_below > 0 && qlen >= q_below)) return;
    const int slot = state_slots[s];
    if (slot < 0 || slot >= num_slots) {
        if (threadIdx.x == 0 && status) atomicExch(status, 3);
        return;
    }
    const float decay = powers[(size_t)h * (FD_C + 1) + 1];
    const bool wide_x = wide & 1, wide_s = wide & 2;
    float* S_mine = state + (size_t)slot * slot_stride + ((size_t)h * cols + col0) * rows + r0;
    pdl_wait();
    float S[NC][RPL];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < RPL; j += 4) {
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            const float* p = S_mine + (size_t)c * rows + j;
            const int left = col0 + c < cols ? rows - (r0 + j) : 0;
            if (wide_s) { if (left > 0) x = *reinterpret_cast<const float4*>(p); }
            else {
                if (left > 0) x.x = p[0];
                if (left > 1) x.y = p[1];
                if (left > 2) x.z = p[2];
                if (left > 3) x.w = p[3];
            }
            S[c][j] = x.x, S[c][j + 1] = x.y, S[c][j + 2] = x.z, S[c][j + 3] = x.w;
        }
    FdRaw4<T> nk[TG][RPL / 4], nq[TG][RPL / 4], nv[TG][NC / 4];
    auto fetch = [&](int first) {
#pragma unroll
        for (int u = 0; u < TG; ++u) {
            const bool ok = first + u < qlen;
            const T* row = qkv + (size_t)(t0 + first + u) * qkv_stride;
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                const int left = ok ? rows - (r0 + 4 * j) : 0;
                nk[u][j] = fd_load4<T>(row + k_off + (size_t)h * rows + r0 + 4 * j, left, wide_x);
                nq[u][j] = fd_load4<T>(row + q_off + (size_t)h * rows + r0 + 4 * j, left, wide_x);
            }
#pragma unroll
            for (int j = 0; j < NC / 4; ++j)
                nv[u][j] = fd_load4<T>(row + v_off + (size_t)h * cols + col0 + 4 * j, ok ? cols - (col0 + 4 * j) : 0, wide_x);
        }
    };
    fetch(0);
    if (positions[t0] == 0) {
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int j = 0; j < RPL; ++j) S[c][j] = 0.f;
    }
    // after the exchange this lane holds the sum of column `mine` of its group
    const int mine = sl / (LPC / NC);
    const bool writes = sl % (LPC / NC) == 0 && col0 + mine < cols;
    for (int first = 0; first < qlen; first += TG) {
        FdRaw4<T> ck[TG][RPL / 4], cq[TG][RPL / 4], cv[TG][NC / 4];
#pragma unroll
        for (int u = 0; u < TG; ++u) {
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) { ck[u][j] = nk[u][j]; cq[u][j] = nq[u][j]; }
#pragma unroll
            for (int j = 0; j < NC / 4; ++j) cv[u][j] = nv[u][j];
        }
        if (first + TG < qlen) fetch(first + TG);
#pragma unroll
        for (int u = 0; u < TG; ++u) {
            if (first + u >= qlen) break;                               // (the same for the whole block)
            float part[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) part[c] = 0.f;
            float vv[NC];
#pragma unroll
            for (int j = 0; j < NC / 4; ++j) {
                const float4 v = fd_act4(cv[u][j].f32(), act);
                vv[4 * j] = v.x, vv[4 * j + 1] = v.y, vv[4 * j + 2] = v.z, vv[4 * j + 3] = v.w;
            }
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                const float4 k = fd_act4(ck[u][j].f32(), act), q = fd_act4(cq[u][j].f32(), act);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    float* x = S[c] + 4 * j;
                    x[0] = fmaf(k.x, vv[c], decay * x[0]);
                    x[1] = fmaf(k.y, vv[c], decay * x[1]);
                    x[2] = fmaf(k.z, vv[c], decay * x[2]);
                    x[3] = fmaf(k.w, vv[c], decay * x[3]);
                    part[c] += fmaf(x[0], q.x, x[1] * q.y) + fmaf(x[2], q.z, x[3] * q.w);
                }
            }
            // halves of the sums change places until a lane holds one; then the rest of the lanes of a column add up
            int off = LPC / 2;
#pragma unroll
            for (int n = NC / 2; n >= 1; n >>= 1, off >>= 1) {
                const bool upper = sl & off;
#pragma unroll
                for (int c = 0; c < n; ++c) {
                    const float give = upper ? part[c] : part[c + n];
                    const float keep = upper ? part[c + n] : part[c];
                    part[c] = keep + __shfl_xor_sync(0xffffffffu, give, off);
                }
            }
#pragma unroll
            for (; off > 0; off >>= 1) part[0] += __shfl_xor_sync(0xffffffffu, part[0], off);
            if (writes) out[((size_t)(t0 + first + u) * nh + h) * cols + col0 + mine] = q_scale * part[0];
        }
    }
    pdl_trigger();
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < RPL; j += 4) {
            float* p = S_mine + (size_t)c * rows + j;
            const int left = col0 + c < cols ? rows - (r0 + j) : 0;
            if (wide_s) { if (left > 0) *reinterpret_cast<float4*>(p) = make_float4(S[c][j], S[c][j + 1], S[c][j + 2], S[c][j + 3]); }
            else {
                if (left > 0) p[0] = S[c][j];
                if (left > 1) p[1] = S[c][j + 1];
                if (left > 2) p[2] = S[c][j + 2];
                if (left > 3) p[3] = S[c][j + 3];
            }
        }
}

// ---- chunks ----------------------------------------------------------------------------------------------
constexpr int FD_CT = 256;         // threads of a block of either kernel
constexpr int FD_CB = 64;          // columns of S a block of the first kernel owns; of the second too
constexpr int FD_RB = 32;          // rows of S a block of the first kernel owns (a warp: 16 columns x 16 rows)
constexpr int FD_VLD = FD_CB + 8, FD_KLD = FD_RB + 8;       // shared rows end 16 bytes further: ldmatrix without bank conflicts

// eight bfloat16 numbers, through SiLU when asked for
__device__ __forceinline__ void fd_unpack8(const uint4& raw, float (&f)[8], int act) {
    const unsigned w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
        f[2 * i] = act ? fd_silu_16(x.x) : x.x;
        f[2 * i + 1] = act ? fd_silu_16(x.y) : x.y;
    }
}
__device__ __forceinline__ uint4 fd_act8(const uint4& raw, int act) {
    if (!act) return raw;
    float f[8];
    fd_unpack8(raw, f, act);
    return make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}
// a pair of floats as two pairs of bfloat16 whose sums they are, to 16 bits
__device__ __forceinline__ void fd_split(float a, float b, unsigned& hi, unsigned& lo) {
    const __nv_bfloat162 x = __floats2bfloat162_rn(a, b);
    const float2 back = __bfloat1622float2(x);
    hi = *reinterpret_cast<const unsigned*>(&x);
    lo = pack_bf16(a - back.x, b - back.y);
}
// chunks of the sequences before s that take the chunked form
__device__ __forceinline__ int fd_chunks_before(const int* __restrict__ cu_q, int s, int min_q) {
    const int lane = threadIdx.x & 31;
    int sum = 0;
    for (int i = lane; i < s; i += 32) {
        const int len = cu_q[i + 1] - cu_q[i];
        if (len >= min_q) sum += (len + FD_C - 1) / FD_C;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    return sum;
}

// Walks the chunks of one (sequence, head) for a part of S (FD_CB columns x FD_RB rows).  A warp's accumulators are S^T:
// 16 columns x 16 rows, in two tiles of eight rows.
__global__ void __launch_bounds__(FD_CT)
fixed_decay_states_kernel(const __nv_bfloat16* __restrict__ qkv, long long qkv_stride, int k_off, int v_off,
                          const float* __restrict__ powers, int act, float* __restrict__ state, long long slot_stride,
                          const int* __restrict__ state_slots, const int* __restrict__ cu_q, const int* __restrict__ positions,
                          uint4* __restrict__ scratch, int scratch_chunks, int nh, int rows, int cols, int num_slots, int min_q,
                          int* __restrict__ status) {
    __shared__ __align__(16) __nv_bfloat16 sV[FD_C * FD_VLD], sKh[FD_C * FD_KLD], sKl[FD_C * FD_KLD];
    __shared__ float pw[FD_C + 1];
    constexpr int VP = FD_C * FD_CB / 8 / FD_CT, KP = FD_C * FD_RB / 8 / FD_CT;      // 16-byte pieces a thread brings
    const int s = blockIdx.z, h = blockIdx.y;
    const int rblocks = (rows + FD_RB - 1) / FD_RB;
    const int col0 = (blockIdx.x / rblocks) * FD_CB, row0 = (blockIdx.x % rblocks) * FD_RB;
    const int wc = (threadIdx.x >> 5) & 3, wr = threadIdx.x >> 7, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int t0 = cu_q[s], qlen = cu_q[s + 1] - t0;
    if (qlen < min_q) return;
    const int slot = state_slots[s];
    const int chunks = (qlen + FD_C - 1) / FD_C;
    const int base = fd_chunks_before(cu_q, s, min_q);
    if (slot < 0 || slot >= num_slots || base + chunks > scratch_chunks) {
        if (threadIdx.x == 0 && status) atomicExch(status, 3);
        return;
    }
    for (int i = threadIdx.x; i <= FD_C; i += FD_CT) pw[i] = powers[(size_t)h * (FD_C + 1) + i];
    const int KS = (rows + 15) / 16, CT = (cols + 7) / 8;
    pdl_wait();
    const bool fresh = positions[t0] == 0;

    float acc[2][4];
    float* S_glob = state + (size_t)slot * slot_stride + (size_t)h * cols * rows;
    const int ca = col0 + wc * 16 + g;                      // this lane's columns: ca and ca + 8
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
        const int r = row0 + wr * 16 + nt * 8 + 2 * t;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int c = ca + 8 * half;
            float2 x = make_float2(0.f, 0.f);
            if (!fresh && c < cols && r < rows) x = *reinterpret_cast<const float2*>(S_glob + (size_t)c * rows + r);
            acc[nt][2 * half] = x.x;
            acc[nt][2 * half + 1] = x.y;
        }
    }

    uint4 rv[VP], rk[KP];
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    auto fetch = [&](int c) {
        const int first = c * FD_C, L = min(FD_C, qlen - first);
        const __nv_bfloat16* at = qkv + (size_t)(t0 + first) * qkv_stride;
#pragma unroll
        for (int i = 0; i < VP; ++i) {
            const int idx = threadIdx.x + i * FD_CT, tok = idx / (FD_CB / 8), cc = col0 + (idx % (FD_CB / 8)) * 8;
            rv[i] = tok < L && cc < cols ? *reinterpret_cast<const uint4*>(at + (size_t)tok * qkv_stride + v_off + (size_t)h * cols + cc) : zero;
        }
#pragma unroll
        for (int i = 0; i < KP; ++i) {
            const int idx = threadIdx.x + i * FD_CT, tok = idx / (FD_RB / 8), rr = row0 + (idx % (FD_RB / 8)) * 8;
            rk[i] = tok < L && rr < rows ? *reinterpret_cast<const uint4*>(at + (size_t)tok * qkv_stride + k_off + (size_t)h * rows + rr) : zero;
        }
    };
    fetch(0);
    const int mat = lane >> 3, rin = lane & 7;
    for (int c = 0; c < chunks; ++c) {
        const int L = min(FD_C, qlen - c * FD_C);
        __syncthreads();                                      // the products of the chunk before have read shared memory
#pragma unroll
        for (int i = 0; i < VP; ++i) {
            const int idx = threadIdx.x + i * FD_CT, tok = idx / (FD_CB / 8), piece = idx % (FD_CB / 8);
            *reinterpret_cast<uint4*>(sV + tok * FD_VLD + piece * 8) = fd_act8(rv[i], act);
        }
#pragma unroll
        for (int i = 0; i < KP; ++i) {
            const int idx = threadIdx.x + i * FD_CT, tok = idx / (FD_RB / 8), piece = idx % (FD_RB / 8);
            const float p = pw[max(L - 1 - tok, 0)];          // (tokens behind the chunk are rows of zeros)
            float f[8];
            fd_unpack8(rk[i], f, act);
            uint4 hi, lo;
            fd_split(f[0] * p, f[1] * p, hi.x, lo.x);
            fd_split(f[2] * p, f[3] * p, hi.y, lo.y);
            fd_split(f[4] * p, f[5] * p, hi.z, lo.z);
            fd_split(f[6] * p, f[7] * p, hi.w, lo.w);
            *reinterpret_cast<uint4*>(sKh + tok * FD_KLD + piece * 8) = hi;
            *reinterpret_cast<uint4*>(sKl + tok * FD_KLD + piece * 8) = lo;
        }
        __syncthreads();
        if (c + 1 < chunks) fetch(c + 1);                     // in flight while the products run
        if (c > 0 || !fresh) {                                // (a fresh sequence's first chunk has no state before it)
            uint4* dst = scratch + ((size_t)(base + c) * nh + h) * ((size_t)KS * CT * 32);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int ct = (col0 + wc * 16) / 8 + half, ks = row0 / 16 + wr;
                if (ct < CT && ks < KS) {
                    uint4 w;
                    fd_split(acc[0][2 * half], acc[0][2 * half + 1], w.x, w.z);
                    fd_split(acc[1][2 * half], acc[1][2 * half + 1], w.y, w.w);
                    dst[((size_t)ct * KS + ks) * 32 + lane] = w;
                }
            }
        }
        const float pl = pw[L];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[nt][i] *= pl;
        const int ksteps = (L + 15) / 16;
#pragma unroll 4
        for (int kt = 0; kt < ksteps; ++kt) {
            unsigned a[4];
            ldmatrix_x4_trans(a[0], a[1], a[2], a[3], sV + (kt * 16 + (mat >> 1) * 8 + rin) * FD_VLD + wc * 16 + (mat & 1) * 8);
            const int at = (kt * 16 + (mat & 1) * 8 + rin) * FD_KLD + wr * 16 + (mat >> 1) * 8;
            unsigned b0, b1, b2, b3;
            ldmatrix_x4_trans(b0, b1, b2, b3, sKh + at);
            mma_bf16_16816(acc[0], a, b0, b1);
            mma_bf16_16816(acc[1], a, b2, b3);
            ldmatrix_x4_trans(b0, b1, b2, b3, sKl + at);
            mma_bf16_16816(acc[0], a, b0, b1);
            mma_bf16_16816(acc[1], a, b2, b3);
        }
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
        const int r = row0 + wr * 16 + nt * 8 + 2 * t;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int c = ca + 8 * half;
            if (c < cols && r < rows) *reinterpret_cast<float2*>(S_glob + (size_t)c * rows + r) = make_float2(acc[nt][2 * half], acc[nt][2 * half + 1]);
        }
    }
}

// One chunk of one (sequence, head), FD_CB columns of the output.  A warp owns 16 tokens; which 16 is arranged so that
// the two warps of a scheduler together meet the same number of earlier tokens as any other two.
__global__ void __launch_bounds__(FD_CT, 2)
fixed_decay_output_kernel(const __nv_bfloat16* __restrict__ qkv, long long qkv_stride, int q_off, int k_off, int v_off,
                          const float* __restrict__ powers, float q_scale, int act, const int* __restrict__ state_slots,
                          const int* __restrict__ cu_q, const int* __restrict__ positions, const uint4* __restrict__ scratch,
                          int scratch_chunks, float* __restrict__ out, int nh, int rows, int cols, int num_slots, int min_q) {
    extern __shared__ __align__(16) unsigned char fd_smem[];
    const int KS = (rows + 15) / 16, CT = (cols + 7) / 8, ld = KS * 16 + 8;
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(fd_smem);
    __nv_bfloat16* sK = sQ + FD_C * ld;
    __nv_bfloat16* sV = sK + FD_C * ld;
    float* pw = reinterpret_cast<float*>(sV + FD_C * FD_VLD);
    const int s = blockIdx.z, h = blockIdx.y;
    const int slices = (cols + FD_CB - 1) / FD_CB;
    const int c = blockIdx.x / slices, col0 = (blockIdx.x % slices) * FD_CB;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    pdl_trigger();
    const int t0 = cu_q[s], qlen = cu_q[s + 1] - t0;
    if (qlen < min_q || c * FD_C >= qlen) return;
    const int slot = state_slots[s];
    const int base = fd_chunks_before(cu_q, s, min_q);
    if (slot < 0 || slot >= num_slots || base + (qlen + FD_C - 1) / FD_C > scratch_chunks) return;     // (the first kernel has said so)
    const int L = min(FD_C, qlen - c * FD_C);
    for (int i = threadIdx.x; i <= FD_C; i += FD_CT) pw[i] = powers[(size_t)h * (FD_C + 1) + i];
    pdl_wait();
    const bool has_state = c > 0 || positions[t0] != 0;
    const __nv_bfloat16* at = qkv + (size_t)(t0 + c * FD_C) * qkv_stride;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    const int pieces = KS * 2;                                // 16-byte pieces of a row of q or k
    const int LT = (L + 15) & ~15;                            // rows that the tiles read
    constexpr int IN = 4;                                     // pieces of q and of k a thread has in flight
    for (int i0 = 0; i0 < LT * pieces; i0 += IN * FD_CT) {
        uint4 qv[IN], kv[IN];
        int to[IN];
#pragma unroll
        for (int i = 0; i < IN; ++i) {
            const int idx = i0 + i * FD_CT + threadIdx.x;
            const int tok = idx / pieces, r = (idx - tok * pieces) * 8;
            const bool ok = tok < L && r < rows;
            const __nv_bfloat16* p = at + (size_t)tok * qkv_stride + (size_t)h * rows + r;
            qv[i] = ok ? *reinterpret_cast<const uint4*>(p + q_off) : zero;
            kv[i] = ok ? *reinterpret_cast<const uint4*>(p + k_off) : zero;
            to[i] = tok < LT ? tok * ld + r : -1;
        }
#pragma unroll
        for (int i = 0; i < IN; ++i) {
            if (to[i] < 0) continue;
            *reinterpret_cast<uint4*>(sQ + to[i]) = fd_act8(qv[i], act);
            *reinterpret_cast<uint4*>(sK + to[i]) = fd_act8(kv[i], act);
        }
    }
#pragma unroll
    for (int i = 0; i < FD_C * FD_CB / 8 / FD_CT; ++i) {
        const int idx = threadIdx.x + i * FD_CT, tok = idx / (FD_CB / 8), cc = (idx % (FD_CB / 8)) * 8;
        const uint4 vv = tok < L && col0 + cc < cols ? *reinterpret_cast<const uint4*>(at + (size_t)tok * qkv_stride + v_off + (size_t)h * cols + col0 + cc) : zero;
        *reinterpret_cast<uint4*>(sV + tok * FD_VLD + cc) = fd_act8(vv, act);
    }
    const int mt = warp < 4 ? warp : 11 - warp;               // (warps w and w + 4 share a scheduler)
    const bool on = mt * 16 < LT;
    const int mat = lane >> 3, rin = lane & 7;
    // the state's first operands are on their way while the others finish loading
    const uint4* src = scratch + ((size_t)(base + c) * nh + h) * ((size_t)KS * CT * 32) + lane;
    const int ct0 = col0 / 8;
    uint4 f[8];
    auto load_s = [&](int ks) {
#pragma unroll
        for (int n = 0; n < 8; ++n) f[n] = ct0 + n < CT ? src[((size_t)(ct0 + n) * KS + ks) * 32] : zero;
    };
    if (has_state && on) load_s(0);
    __syncthreads();
    if (!on) return;
    float o[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    const __nv_bfloat16* q_mine = sQ + (mt * 16 + (mat & 1) * 8 + rin) * ld + (mat >> 1) * 8;
    if (has_state) {
        for (int ks = 0; ks < KS; ++ks) {
            uint4 w[8];
#pragma unroll
            for (int n = 0; n < 8; ++n) w[n] = f[n];
            if (ks + 1 < KS) load_s(ks + 1);
            unsigned a[4];
            ldmatrix_x4(a[0], a[1], a[2], a[3], q_mine + ks * 16);
#pragma unroll
            for (int n = 0; n < 8; ++n) mma_bf16_16816(o[n], a, w[n].x, w[n].y);
#pragma unroll
            for (int n = 0; n < 8; ++n) mma_bf16_16816(o[n], a, w[n].z, w[n].w);
        }
        const float pa = pw[mt * 16 + g + 1], pb = pw[mt * 16 + g + 9];
#pragma unroll
        for (int n = 0; n < 8; ++n) { o[n][0] *= pa; o[n][1] *= pa; o[n][2] *= pb; o[n][3] *= pb; }
    }
    for (int jb = 0; jb <= mt; ++jb) {                        // sixteen earlier tokens at a time
        // (even and odd steps of the inner size add up apart: two chains instead of one)
        float a[2][2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) a[0][n][e] = a[1][n][e] = 0.f;
        const __nv_bfloat16* k_mine = sK + (jb * 16 + (mat >> 1) * 8 + rin) * ld + (mat & 1) * 8;
        for (int ks = 0; ks < KS; ks += 2) {
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                if (ks + x >= KS) break;
                unsigned q[4], b0, b1, b2, b3;
                ldmatrix_x4(q[0], q[1], q[2], q[3], q_mine + (ks + x) * 16);
                ldmatrix_x4(b0, b1, b2, b3, k_mine + (ks + x) * 16);
                mma_bf16_16816(a[x][0], q, b0, b1);
                mma_bf16_16816(a[x][1], q, b2, b3);
            }
        }
        unsigned hi[4], lo[4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {                     // rows g and g + 8 of the tile
                const int d = mt * 16 + g + 8 * e - (jb * 16 + n * 8 + 2 * t);              // how far back the first of the pair lies
                const float x = d >= 0 ? (a[0][n][2 * e] + a[1][n][2 * e]) * pw[max(d, 0)] : 0.f;
                const float y = d >= 1 ? (a[0][n][2 * e + 1] + a[1][n][2 * e + 1]) * pw[max(d - 1, 0)] : 0.f;
                fd_split(x, y, hi[2 * n + e], lo[2 * n + e]);
            }
        unsigned b[4][4];
#pragma unroll
        for (int nn = 0; nn < 4; ++nn)
            ldmatrix_x4_trans(b[nn][0], b[nn][1], b[nn][2], b[nn][3], sV + (jb * 16 + (mat & 1) * 8 + rin) * FD_VLD + nn * 16 + (mat >> 1) * 8);
#pragma unroll
        for (int nn = 0; nn < 4; ++nn) {
            mma_bf16_16816(o[2 * nn], hi, b[nn][0], b[nn][1]);
            mma_bf16_16816(o[2 * nn + 1], hi, b[nn][2], b[nn][3]);
        }
#pragma unroll
        for (int nn = 0; nn < 4; ++nn) {
            mma_bf16_16816(o[2 * nn], lo, b[nn][0], b[nn][1]);
            mma_bf16_16816(o[2 * nn + 1], lo, b[nn][2], b[nn][3]);
        }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int i = mt * 16 + g + 8 * e;
        if (i >= L) continue;
        float* row = out + ((size_t)(t0 + c * FD_C + i) * nh + h) * cols + col0 + 2 * t;
#pragma unroll
        for (int n = 0; n < 8; ++n)
            if (col0 + n * 8 < cols) *reinterpret_cast<float2*>(row + n * 8) = make_float2(q_scale * o[n][2 * e], q_scale * o[n][2 * e + 1]);
    }
}

VAPI_EXPORT int vapi_fixed_decay_chunk() { return FD_C; }

// 16-byte words of scratch memory that one chunk takes (0: these sizes have no chunked form)
VAPI_EXPORT long long vapi_fixed_decay_chunk_words(int nh, int rows, int cols) {
    if (rows <= 0 || rows > 256 || rows % 8 || cols <= 0 || cols % 8) return 0;
    return (long long)nh * ((rows + 15) / 16) * ((cols + 7) / 8) * 32;
}

// qkv [n, *]: q heads [nh, rows] at q_off, k heads [nh, rows] at k_off, v heads [nh, cols] at v_off of a row of `qkv_stride`
// elements; powers [nh, FD_C + 1]; state [slots, *] with S [nh, cols, rows] in front; out [n, nh * cols] float.
// scratch (with scratch_chunks chunks): sequences of min_q tokens or more take the chunked form.  null: all walk.
VAPI_EXPORT int vapi_fixed_decay(const void* qkv, long long qkv_stride, int q_off, int k_off, int v_off, int dtype,
                                 const float* powers, float q_scale, int act, float* state, long long slot_stride,
                                 const int* state_slots, const int* cu_q, const int* positions, float* out, int num_seqs, int nh,
                                 int rows, int cols, int num_slots, int max_q, void* scratch, int scratch_chunks, int min_q,
                                 int* status, cudaStream_t stream) {
    if (num_seqs <= 0) return 0;
    if (nh <= 0 || rows <= 0 || rows > 256 || cols <= 0) return fail(-1, "fixed_decay: %d heads, state %d x %d (rows up to 256)", nh, rows, cols);
    if (dtype != VAPI_F32 && dtype != VAPI_BF16) return fail(-2, "fixed_decay: unsupported dtype %d", dtype);
    if (nh > 65535 || num_seqs > 65535) return fail(-1, "fixed_decay: %d heads x %d sequences are too many", nh, num_seqs);
    const bool chunked = scratch != nullptr && max_q >= min_q;
    const size_t esz = dtype == VAPI_F32 ? 4 : 2;
    if (chunked) {
        if (dtype != VAPI_BF16 || vapi_fixed_decay_chunk_words(nh, rows, cols) == 0 || min_q < 1 || scratch_chunks <= 0)
            return fail(-1, "fixed_decay: no chunked form for states of %d x %d, dtype %d", rows, cols, dtype);
        if (q_off % 8 || k_off % 8 || v_off % 8 || qkv_stride % 8 || ((uintptr_t)qkv & 15) || ((uintptr_t)scratch & 15) ||
            slot_stride % 2 || ((uintptr_t)state & 7) || ((uintptr_t)out & 7))
            return fail(-1, "fixed_decay: the chunked form needs 16-byte aligned rows");
        dim3 grid(((cols + FD_CB - 1) / FD_CB) * ((rows + FD_RB - 1) / FD_RB), nh, num_seqs);
        cudaError_t e = launch_if(false, fixed_decay_states_kernel, grid, FD_CT, 0, stream, (const __nv_bfloat16*)qkv, qkv_stride,
                                  k_off, v_off, powers, act, state, slot_stride, state_slots, cu_q, positions, (uint4*)scratch,
                                  scratch_chunks, nh, rows, cols, num_slots, min_q, status);
        int rc = check_launch("fixed_decay (states)", e);
        if (rc != 0) return rc;
        const int ld = ((rows + 15) / 16) * 16 + 8;
        const size_t smem = (size_t)FD_C * (2 * ld + FD_VLD) * 2 + (FD_C + 1) * sizeof(float);
        static size_t allowed = 48 * 1024;
        if (smem > allowed) {
            if (cudaFuncSetAttribute(fixed_decay_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
                return fail(-3, "fixed_decay: %zu bytes of shared memory are not available", smem);
            allowed = smem;
        }
        const long long bx = (long long)((max_q + FD_C - 1) / FD_C) * ((cols + FD_CB - 1) / FD_CB);
        if (bx > 0x7fffffffLL) return fail(-1, "fixed_decay: %d tokens are too many", max_q);
        e = launch(fixed_decay_output_kernel, dim3((unsigned)bx, nh, num_seqs), FD_CT, smem, stream, (const __nv_bfloat16*)qkv,
                   qkv_stride, q_off, k_off, v_off, powers, q_scale, act, state_slots, cu_q, positions, (const uint4*)scratch,
                   scratch_chunks, out, nh, rows, cols, num_slots, min_q);
        rc = check_launch("fixed_decay (output)", e);
        if (rc != 0 || num_seqs == 1) return rc;              // (max_q >= min_q: the only sequence is done)
    }
    // 16-byte (float) / 8-byte (bfloat16) loads of the vectors; 16-byte accesses of the state
    int wide = rows % 4 == 0 && cols % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 && qkv_stride % 4 == 0 &&
               (uintptr_t)qkv % (4 * esz) == 0;
    if (rows % 4 == 0 && slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0) wide |= 2;
    const int q_below = chunked ? min_q : 0;
    cudaError_t e = cudaSuccess;
    const bool early = max_q < 16;
#define FD_WALK_(T, RPL, LPC, NC, TG)                                                                                         \
    e = launch_if(early, fixed_decay_walk_kernel<T, RPL, LPC, NC, TG>, dim3((cols + (32 / LPC) * NC * 4 - 1) / ((32 / LPC) * NC * 4), nh, num_seqs), \
                  FD_THREADS, 0, stream, (const T*)qkv, qkv_stride, q_off, k_off, v_off, powers, q_scale, act, state,         \
                  slot_stride, state_slots, cu_q, positions, out, nh, rows, cols, num_slots, q_below, wide, status)
#define FD_WALK(T, RPL, LPC, NC) do { if (max_q == 1) FD_WALK_(T, RPL, LPC, NC, 1); else FD_WALK_(T, RPL, LPC, NC, sizeof(T) == 4 ? 2 : 4); } while (0)
#define FD_SIZES(T)                                                                                                           \
    do {                                                                                                                      \
        if (rows <= 32) FD_WALK(T, 4, 8, 4);                                                                                  \
        else if (rows <= 64) FD_WALK(T, 4, 16, 4);                                                                            \
        else if (rows <= 128) { if (many) FD_WALK(T, 4, 32, 8); else FD_WALK(T, 4, 32, 4); }                                  \
        else FD_WALK(T, 8, 32, 4);                                                                                            \
    } while (0)
    const bool many = (long long)((cols + 31) / 32) * nh * num_seqs >= 2LL * sm_count();
    if (dtype == VAPI_F32) FD_SIZES(float);
    else FD_SIZES(__nv_bfloat16);
#undef FD_SIZES
#undef FD_WALK
#undef FD_WALK_
    return check_launch("fixed_decay (walk)", e);
}

VAPI_EXPORT const char* vapi_last_error() { return error_buffer(); }
