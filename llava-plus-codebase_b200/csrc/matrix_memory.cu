// Matrix memories of the layer-list decoders whose decay is ONE number per head and token (kernels.h, MemoryArgs): the gated delta rule and
// the mLSTM memory with exponential gates. A portion of a prompt (n rows of one slot) and a decode step (one row of each of B slots) take
// the same kernel; rows come as segments, a segment at position 0 starts from an empty memory whatever its slot held.
//
// Eight lanes share a value column and hold its keys' state in registers (KPT each), a warp walks 4 columns, a CTA 16. Tokens come in
// tiles: q, k, v and the raw gates of the next tile are on their way into shared memory (cp.async) while the current one is walked, and
// what a token needs besides its vectors (unit norms and k . q of the delta rule, decay and write strength, the running maximum) is made
// once per tile and head. Both dot products of the delta rule run against the state BEFORE the token: with a = S^T k and b = S^T q,
//     u = beta (v - g a),   S' = g S + k u^T,   y = g b + u (k . q),
// so only the sum a over a column's eight lanes is on the chain from token to token; the read-outs' sums b meet once per four tokens. State,
// gates and sums are fp32.
#include "common.cuh"
#include "kernels.h"

namespace b2 {
namespace {

constexpr int MM_TT = 32, MM_L = 8, MM_WARPS = 4, MM_COLS = MM_WARPS * 32 / MM_L, MM_THREADS = MM_WARPS * 32;

__device__ __forceinline__ float mm_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float mm_log_sigmoid(float v) { return fminf(v, 0.f) - log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ void cp_async_16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ float sum8(float v) {   // over the eight lanes of a column
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 4);
}
__device__ __forceinline__ float sum32(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// VEC: dk % 4 == 0 and q / k rows are 16-byte aligned
template <int MODE, int KPT, bool VEC>
__global__ void __launch_bounds__(MM_THREADS) matrix_memory_kernel(MemoryArgs a) {
    constexpr int DKP = KPT * MM_L;                      // keys a CTA holds (the ones past dk stay zero)
    extern __shared__ __align__(16) float sm[];
    float* sQ = sm;                                      // [2][TT][DKP]
    float* sK = sQ + 2 * MM_TT * DKP;                    // [2][TT][DKP]
    float* sV = sK + 2 * MM_TT * DKP;                    // [2][TT][COLS]
    float* sG = sV + 2 * MM_TT * MM_COLS;                // [2][2][TT] raw gates
    float4* sC = reinterpret_cast<float4*>(sG + 4 * MM_TT);   // [TT][2] per-token factors
    float* sO = reinterpret_cast<float*>(sC + 2 * MM_TT);     // [TT][COLS]
    const SeqSeg sg = a.segs[blockIdx.z];
    if (sg.n <= 0) return;
    const int h = blockIdx.y, g = h / (a.heads / a.kv_heads), col0 = blockIdx.x * MM_COLS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & (MM_L - 1), c = warp * (32 / MM_L) + lane / MM_L, col = col0 + c;
    const int dk = a.dk, dv = a.dv, ncol = MODE == MEM_MLSTM ? dv + 1 : dv;
    const float* qg = a.q + (size_t)sg.row0 * a.ldq + (size_t)g * dk;
    const float* kg = a.k + (size_t)sg.row0 * a.ldk + (size_t)g * dk;
    const float* vg = a.v + (size_t)sg.row0 * a.ldv + (size_t)h * dv;
    const float* g1 = a.gate1 + (size_t)sg.row0 * a.ldg + h;
    const float* g2 = a.gate2 + (size_t)sg.row0 * a.ldg + h;

    // keys of a lane: 4 consecutive ones out of every 4 * MM_L, so that the eight lanes of a column read 128 adjoining bytes
    auto key_of = [&](int i) { return (i >> 2) * (4 * MM_L) + l * 4 + (i & 3); };
    float S[KPT];
    float* st = a.state + (((size_t)sg.slot * a.heads + h) * ncol + col) * dk;
    const bool live = col < ncol, load = live && sg.pos0 > 0;
#pragma unroll
    for (int i = 0; i < KPT; i += 4) {
        const int key = key_of(i);
        if (VEC) {
            const float4 v = (load && key < dk) ? *reinterpret_cast<const float4*>(st + key) : make_float4(0.f, 0.f, 0.f, 0.f);
            S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) S[i + e] = (load && key + e < dk) ? st[key + e] : 0.f;
        }
    }
    float* rm = MODE == MEM_MLSTM ? a.run_max + ((size_t)sg.slot * a.heads + h) * gridDim.x + blockIdx.x : nullptr;
    float m_run = (MODE == MEM_MLSTM && sg.pos0 > 0) ? rm[0] : 0.f;   // tracked by warp 0
    const float b1 = a.bias1 != nullptr ? a.bias1[h] : 0.f, b2 = a.bias2 != nullptr ? a.bias2[h] : 0.f;
    const float neg_a = MODE == MEM_DELTA ? -expf(a.a_log[h]) : 0.f;

    // entries that no copy ever writes: padded keys, columns past the last value (the normaliser's column reads 1)
    for (int e = tid; e < 2 * MM_TT * (DKP - dk); e += MM_THREADS) {
        const int t = e / (DKP - dk), key = dk + e % (DKP - dk);
        sQ[t * DKP + key] = 0.f; sK[t * DKP + key] = 0.f;
    }
    for (int e = tid; e < 2 * MM_TT * MM_COLS; e += MM_THREADS) {
        const int cc = col0 + e % MM_COLS;
        if (cc >= dv) sV[e] = (MODE == MEM_MLSTM && cc == dv) ? 1.f : 0.f;
    }
    auto fetch = [&](int t0, int buf) {
        const int nt = min(MM_TT, sg.n - t0);
        float* q = sQ + buf * MM_TT * DKP;
        float* k = sK + buf * MM_TT * DKP;
        if (VEC) {
            const int n4 = dk >> 2;
            for (int e = tid; e < nt * n4; e += MM_THREADS) {
                const int t = e / n4, d = (e - t * n4) * 4;
                cp_async_16(q + t * DKP + d, qg + (size_t)(t0 + t) * a.ldq + d);
                cp_async_16(k + t * DKP + d, kg + (size_t)(t0 + t) * a.ldk + d);
            }
        } else {
            for (int e = tid; e < nt * dk; e += MM_THREADS) {
                const int t = e / dk, d = e - t * dk;
                cp_async_4(q + t * DKP + d, qg + (size_t)(t0 + t) * a.ldq + d);
                cp_async_4(k + t * DKP + d, kg + (size_t)(t0 + t) * a.ldk + d);
            }
        }
        float* v = sV + buf * MM_TT * MM_COLS;
        for (int e = tid; e < nt * MM_COLS; e += MM_THREADS) {
            const int t = e / MM_COLS, cc = e % MM_COLS;
            if (col0 + cc < dv) cp_async_4(v + e, vg + (size_t)(t0 + t) * a.ldv + col0 + cc);
        }
        if (tid < 2 * MM_TT) {
            const int t = tid % MM_TT;
            if (t < nt) cp_async_4(sG + buf * 2 * MM_TT + tid, (tid < MM_TT ? g1 : g2) + (size_t)(t0 + t) * a.ldg);
        }
        cp_async_commit();
    };
    fetch(0, 0);
    int buf = 0;
    for (int t0 = 0; t0 < sg.n; t0 += MM_TT, buf ^= 1) {
        const int nt = min(MM_TT, sg.n - t0);
        cp_async_wait_all();
        __syncthreads();                                      // this tile has landed; the other buffer and sC are free
        if (t0 + MM_TT < sg.n) fetch(t0 + MM_TT, buf ^ 1);
        const float* q = sQ + buf * MM_TT * DKP;
        const float* k = sK + buf * MM_TT * DKP;
        const float* v = sV + buf * MM_TT * MM_COLS;
        const float* raw = sG + buf * 2 * MM_TT;
        if (MODE == MEM_DELTA) {
            // per token: g, beta, g / |k|, g s / |q|, 1 / |k|, s (k . q) / (|k| |q|)
            float sq[MM_TT / MM_WARPS], sk[MM_TT / MM_WARPS], kq[MM_TT / MM_WARPS];
#pragma unroll
            for (int u = 0; u < MM_TT / MM_WARPS; ++u) {
                const int t = warp + u * MM_WARPS;
                sq[u] = 0.f; sk[u] = 0.f; kq[u] = 0.f;
                if (t < nt) {
                    for (int d = lane * 4; d < DKP; d += 128) {
                        const float4 x = *reinterpret_cast<const float4*>(q + t * DKP + d), y = *reinterpret_cast<const float4*>(k + t * DKP + d);
                        sq[u] += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
                        sk[u] += (y.x * y.x + y.y * y.y) + (y.z * y.z + y.w * y.w);
                        kq[u] += (x.x * y.x + x.y * y.y) + (x.z * y.z + x.w * y.w);
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < MM_TT / MM_WARPS; ++u) { sq[u] = sum32(sq[u]); sk[u] = sum32(sk[u]); kq[u] = sum32(kq[u]); }
            float mq = 0.f, mk = 0.f, mkq = 0.f;              // lane u finishes the warp's token u
#pragma unroll
            for (int u = 0; u < MM_TT / MM_WARPS; ++u)
                if (lane == u) { mq = sq[u]; mk = sk[u]; mkq = kq[u]; }
            const int t = warp + lane * MM_WARPS;
            if (lane < MM_TT / MM_WARPS && t < nt) {
                const float rq = a.q_scale / sqrtf(mq + 1e-6f), rk = 1.f / sqrtf(mk + 1e-6f);
                const float beta = 1.f / (1.f + expf(-(raw[t] + b1))), gd = expf(neg_a * mm_softplus(raw[MM_TT + t] + b2));
                sC[2 * t] = make_float4(gd, beta, gd * rk, gd * rq);
                sC[2 * t + 1] = make_float4(rk, mkq * rk * rq, 0.f, 0.f);
            }
        } else if (warp == 0) {
            // per token: decay exp(f + m - m'), write strength exp(i - m'), floor exp(-m'). m' over the tile is a scan of (f, i) pairs:
            // over the tokens up to t, m' = max(F + m, M). The decay is taken from the DIFFERENCE of two running maxima, which is exact
            // where they are close, so the rounding of a long sum of f never enters the memory.
            const int t = lane;
            float iv = -INFINITY, fv = 0.f;
            if (t < nt) {
                iv = a.cap * tanhf((raw[t] + b1) / a.cap);
                fv = mm_log_sigmoid(a.cap * tanhf((raw[MM_TT + t] + b2) / a.cap));
            }
            float Fs = fv, Ms = iv;
#pragma unroll
            for (int o = 1; o < MM_TT; o <<= 1) {
                const float Fl = __shfl_up_sync(0xffffffffu, Fs, o), Ml = __shfl_up_sync(0xffffffffu, Ms, o);
                if (lane >= o) { Ms = fmaxf(Ml + Fs, Ms); Fs += Fl; }
            }
            const float mt = fmaxf(Fs + m_run, Ms);
            float mp = __shfl_up_sync(0xffffffffu, mt, 1);
            if (lane == 0) mp = m_run;
            if (t < nt) sC[2 * t] = make_float4(expf(fv + (mp - mt)), expf(iv - mt), expf(-mt), 0.f);
            m_run = __shfl_sync(0xffffffffu, mt, nt - 1);
        }
        __syncthreads();
        // Tokens go in groups of four: a token's vectors are read one token ahead, and the sums that are not on the chain from token to token
        // (the read-outs) meet once per group, four tokens' worth folded into one value per lane pair.
        float kb[2][KPT], qb[2][KPT];
        auto read = [&](int t, float (&kx)[KPT], float (&qx)[KPT]) {
#pragma unroll
            for (int i = 0; i < KPT; i += 4) {
                const int off = t * DKP + (i >> 2) * (4 * MM_L) + l * 4;
                const float4 x = *reinterpret_cast<const float4*>(k + off), y = *reinterpret_cast<const float4*>(q + off);
                kx[i] = x.x; kx[i + 1] = x.y; kx[i + 2] = x.z; kx[i + 3] = x.w;
                qx[i] = y.x; qx[i + 1] = y.y; qx[i + 2] = y.z; qx[i + 3] = y.w;
            }
        };
        // one token: updates S, returns this lane's share of the read-out's sum; u: what the delta rule writes (before 1 / |k|)
        auto step = [&](int t, const float (&kk)[KPT], const float (&qq)[KPT], float& u) {
            const float4 f0 = sC[2 * t];
            const float vt = v[t * MM_COLS + c];
            float pb[4] = {0.f, 0.f, 0.f, 0.f};
            if (MODE == MEM_DELTA) {
                float pa[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int i = 0; i < KPT; ++i) pa[i & 3] = fmaf(S[i], kk[i], pa[i & 3]);
#pragma unroll
                for (int i = 0; i < KPT; ++i) pb[i & 3] = fmaf(S[i], qq[i], pb[i & 3]);
                const float sa = sum8((pa[0] + pa[1]) + (pa[2] + pa[3]));
                u = f0.y * fmaf(-f0.z, sa, vt);
                const float uk = u * sC[2 * t + 1].x;
#pragma unroll
                for (int i = 0; i < KPT; ++i) S[i] = fmaf(kk[i], uk, f0.x * S[i]);
            } else {
                const float wv = f0.y * vt;
#pragma unroll
                for (int i = 0; i < KPT; ++i) {
                    S[i] = fmaf(f0.x, S[i], kk[i] * wv);
                    pb[i & 3] = fmaf(S[i], qq[i], pb[i & 3]);
                }
            }
            return (pb[0] + pb[1]) + (pb[2] + pb[3]);
        };
        auto finish = [&](int t, float sum, float u) {   // the whole sum of token t's read-out -> its value
            const float4 f0 = sC[2 * t];
            if (MODE == MEM_DELTA) return fmaf(f0.w, sum, u * sC[2 * t + 1].y);
            const float sb = a.q_scale * sum;
            return col == dv ? fmaxf(fabsf(sb), f0.z) + 1e-6f : sb;
        };
        read(0, kb[0], qb[0]);
        int t = 0;
        for (; t + 4 <= nt; t += 4) {
            float p[4], u[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                if (e < 3 || t + 4 < MM_TT) read(t + e + 1, kb[(e + 1) & 1], qb[(e + 1) & 1]);
                p[e] = step(t + e, kb[e & 1], qb[e & 1], u[e]);
            }
            // eight lanes x four sums: lanes with bit 2 set keep tokens 2 and 3, then bit 1 picks one of the two, bit 0 only adds
            const bool hi = (l & 4) != 0, odd = (l & 2) != 0;
            float k0 = hi ? p[2] : p[0], k1 = hi ? p[3] : p[1];
            k0 += __shfl_xor_sync(0xffffffffu, hi ? p[0] : p[2], 4);
            k1 += __shfl_xor_sync(0xffffffffu, hi ? p[1] : p[3], 4);
            float sum = odd ? k1 : k0;
            sum += __shfl_xor_sync(0xffffffffu, odd ? k0 : k1, 2);
            sum += __shfl_xor_sync(0xffffffffu, sum, 1);
            const int tk = t + (hi ? 2 : 0) + (odd ? 1 : 0);
            const float uu = hi ? (odd ? u[3] : u[2]) : (odd ? u[1] : u[0]);
            const float o = finish(tk, sum, uu);
            if ((l & 1) == 0) sO[tk * MM_COLS + c] = o;
        }
        for (; t < nt; ++t) {   // up to three tokens behind the last group
            float u = 0.f;
            const float sum = sum8(step(t, kb[0], qb[0], u));
            if (t + 1 < nt) read(t + 1, kb[0], qb[0]);
            const float o = finish(t, sum, u);
            if (l == 0) sO[t * MM_COLS + c] = o;
        }
        __syncthreads();
        for (int e = tid; e < nt * MM_COLS; e += MM_THREADS) {
            const int t = e / MM_COLS, cc = col0 + e % MM_COLS;
            const size_t row = (size_t)(sg.row0 + t0 + t);
            if (cc < dv) a.y[row * a.ldy + (size_t)h * dv + cc] = sO[e];
            else if (MODE == MEM_MLSTM && cc == dv) a.den[row * a.heads + h] = sO[e];
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < KPT; i += 4) {
            const int key = key_of(i);
            if (VEC) {
                if (key < dk) *reinterpret_cast<float4*>(st + key) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (key + e < dk) st[key + e] = S[i + e];
            }
        }
    }
    if (MODE == MEM_MLSTM && tid == 0) rm[0] = m_run;   // every column block of a head keeps its own copy: no block reads what another writes
}

template <int MODE, int KPT, bool VEC>
int launch_memory(const MemoryArgs& a, cudaStream_t st) {
    const int ncol = a.mode == MEM_MLSTM ? a.dv + 1 : a.dv;
    const size_t smem = ((size_t)4 * MM_TT * KPT * MM_L + 2 * MM_TT * MM_COLS + 4 * MM_TT + 8 * MM_TT + MM_TT * MM_COLS) * sizeof(float);
    if (smem > 48 * 1024) B2_CUDA_CHECK(cudaFuncSetAttribute(matrix_memory_kernel<MODE, KPT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    matrix_memory_kernel<MODE, KPT, VEC><<<dim3(mem_blocks(ncol), a.heads, a.nseg), MM_THREADS, smem, st>>>(a);
    B2_LAUNCH_CHECK();
    return 0;
}
template <int MODE, int KPT>
int launch_memory_k(const MemoryArgs& a, cudaStream_t st) {
    const bool vec = a.dk % 4 == 0 && a.ldq % 4 == 0 && a.ldk % 4 == 0 &&
                     ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k) | reinterpret_cast<uintptr_t>(a.state)) & 15) == 0;
    return vec ? launch_memory<MODE, KPT, true>(a, st) : launch_memory<MODE, KPT, false>(a, st);
}
template <int MODE>
int launch_memory_mode(const MemoryArgs& a, cudaStream_t st) {
    if (a.dk <= 32) return launch_memory_k<MODE, 4>(a, st);
    if (a.dk <= 64) return launch_memory_k<MODE, 8>(a, st);
    if (a.dk <= 128) return launch_memory_k<MODE, 16>(a, st);
    return launch_memory_k<MODE, 32>(a, st);
}
}  // namespace

int mem_blocks(int columns) { return (columns + MM_COLS - 1) / MM_COLS; }

int matrix_memory_f32(const MemoryArgs& a, cudaStream_t st) {
    B2_CHECK_ARG(a.q && a.k && a.v && a.gate1 && a.gate2 && a.state && a.y && a.segs && a.nseg > 0, "matrix_memory: null argument");
    B2_CHECK_ARG(a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dk > 0 && a.dk <= 256 && a.dv > 0, "matrix_memory: heads %d / %d, keys of %d (at most 256), values of %d",
                 a.heads, a.kv_heads, a.dk, a.dv);
    if (a.mode == MEM_DELTA) {
        B2_CHECK_ARG(a.a_log && a.bias2, "matrix_memory(delta): null decay tensor");
        return launch_memory_mode<MEM_DELTA>(a, st);
    }
    B2_CHECK_ARG(a.mode == MEM_MLSTM && a.run_max && a.den && a.cap > 0.f && a.bias1 && a.bias2, "matrix_memory(mlstm): null gate tensor or a non-positive cap");
    return launch_memory_mode<MEM_MLSTM>(a, st);
}

}  // namespace b2
