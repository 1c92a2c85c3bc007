// Row kernels of layers that norm and gate a sublayer's result before it joins the residual stream, whose mixers read
// a mix of a token and the one before it, and which take a learned input per token and layer.  The stream is float32;
// gates, norms, the shift and every sum are float32, and a row's additions have an order that depends on its width only.
//
//   token_shift      out = x + (x' - x) * s per channel, x' the row of the request's token before (its state for the
//                    first token of a step, zero for the first of a sequence); the state becomes the last row.  The
//                    row as it is can be written too, in the compute dtype, for products that read it unshifted.
//   gated_norm_add   x += norm(y * sigmoid(z + zb)) * w,  norm(u) = u / sqrt(mean(u^2) + eps);  y is a product's output
//                    (the unjoined parts of a split K, plus a bias) or the weighted sum of a token's expert rows;
//                    the gate may be absent; the new row can be written in the compute dtype as well.  In steps in
//                    which every request brings one token, the kernel also makes the next layer's token_shift.
//   side_gate        out = gelu_tanh(z) * e,  e a slice of a table's row of the token
//   map_difference   o = a_1 - lambda a_2 per head, divided by its root mean square, times a constant
//   route_chosen     the `top` largest of z + bias per token, and the softmax over those
#include "common.cuh"

__device__ __forceinline__ float4 f4_add(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float shifted_f(float x, float before, float s) { return fmaf(before - x, s, x); }

// ---------------------------------------------------------------------------
// As in a short convolution, only the blocks of a request's first token of the step touch the state: they read it for
// that token and then store the last one's row, so nothing races with the update.
// ---------------------------------------------------------------------------
template <typename O, bool VEC>
__global__ void token_shift_kernel(const float* __restrict__ x, const float* __restrict__ shift, float* __restrict__ state,
                                   O* __restrict__ out, O* __restrict__ plain, const int* __restrict__ q_start,
                                   const int* __restrict__ q_len, const int* __restrict__ slots,
                                   const int* __restrict__ token_req, int D, int max_slots, unsigned* err) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int r = token_req[t], a = q_start[r], n = q_len[r], slot = slots[r];
    const bool first = t == a;
    if (first && (slot < 0 || slot >= max_slots)) {
        if (threadIdx.x == 0) atomicOr(err, AIE_DEV_SLOT_OOB);
        return;
    }
    const float* cur = x + (size_t)t * D;
    const float* prev = first ? state + (size_t)slot * D : cur - D;
    const float* last = x + (size_t)(a + n - 1) * D;
    float* st = state + (size_t)(first ? slot : 0) * D;
    if (VEC) {
        for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4; c < D; c += gridDim.y * blockDim.x * 4) {
            const float4 v = load4<float>(cur + c), b = load4<float>(prev + c), s = load4<float>(shift + c);
            store4<O>(out + (size_t)t * D + c, make_float4(shifted_f(v.x, b.x, s.x), shifted_f(v.y, b.y, s.y),
                                                           shifted_f(v.z, b.z, s.z), shifted_f(v.w, b.w, s.w)));
            if (plain) store4<O>(plain + (size_t)t * D + c, v);
            if (first) store4<float>(st + c, load4<float>(last + c));
        }
    } else {
        for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < D; c += gridDim.y * blockDim.x) {
            const float v = cur[c];
            out[(size_t)t * D + c] = from_f32<O>(shifted_f(v, prev[c], shift[c]));
            if (plain) plain[(size_t)t * D + c] = from_f32<O>(v);
            if (first) st[c] = last[c];
        }
    }
}

extern "C" int aie_token_shift(const float* x, const float* shift, float* state, void* out, void* plain, int out_dtype,
                               const int* q_start, const int* q_len, const int* slots, const int* token_req, int T, int D,
                               int max_slots, unsigned* err, cudaStream_t st) {
    if (T <= 0) return 0;
    if (D <= 0) return AIE_BAD_ARG;
    const bool vec = D % 4 == 0 && !(((size_t)x | (size_t)shift | (size_t)state | (size_t)out | (size_t)plain) & 15);
    const int per = vec ? D / 4 : D, threads = per >= 256 ? 256 : 128;
    int gy = (per + threads - 1) / threads;
    if (gy > 64) gy = 64;
#define GO(O, V)                                                                                                        \
    launch_pdl(token_shift_kernel<O, V>, dim3(T, gy), dim3(threads), 0, st, x, shift, state, (O*)out, (O*)plain, q_start, \
               q_len, slots, token_req, D, max_slots, err)
    if (out_dtype == AIE_F32) {
        if (vec) GO(float, true); else GO(float, false);
    } else if (out_dtype == AIE_BF16) {
        if (vec) GO(bf16, true); else GO(bf16, false);
    } else {
        return AIE_BAD_ARG;
    }
#undef GO
    AIE_LAUNCH_CHECK();
}

// ---------------------------------------------------------------------------
struct BranchSource {
    const float* y;          // parts > 0: [parts, T, D], `stride` floats between parts;  parts == 0: expert rows [rows, D]
    size_t stride;
    int parts;
    const float* bias;       // [D] or null (parts > 0)
    const int* pair_row;     // [T, top]: row of the pair (negative: none)
    const float* weight;     // [T, top]
    int top;
    const float* z;          // gate logits [zparts, T, ldz] or null
    size_t zstride;
    int zparts, ldz;
    const float* zbias;      // [D] or null
};

struct ShiftAhead {          // the next layer's token_shift (out null: not made); every request brings one token
    const float* shift;
    float* state;
    void* out;
    const int* slots;
    const int* token_req;
    int max_slots;
};

// MODE 0: the parts of a product, gate or none;  1: one part each of branch and gate (a step of many tokens);
// 2: expert rows.  Loads of what the previous kernel wrote; the gate's logits come back in g.
template <int MODE>
__device__ __forceinline__ void branch_loads(const BranchSource& b, int t, int c, int D, float4& v, float4& g) {
    if (MODE == 1) {
        v = load4<float>(b.y + (size_t)t * D + c);
        g = load4<float>(b.z + (size_t)t * b.ldz + c);
        return;
    }
    if (b.z) g = load4<float>(b.z + (size_t)t * b.ldz + c);
    if (MODE == 0) {
        const float* p = b.y + (size_t)t * D + c;
        v = load4<float>(p);
#pragma unroll 4
        for (int i = 1; i < b.parts; ++i) v = f4_add(v, load4<float>(p + i * b.stride));
    } else {
        v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int s = 0; s < b.top; ++s) {
            const int row = b.pair_row[(size_t)t * b.top + s];
            const float w = b.weight[(size_t)t * b.top + s];
            const float4 u = row >= 0 ? load4<float>(b.y + (size_t)row * D + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            v = make_float4(fmaf(w, u.x, v.x), fmaf(w, u.y, v.y), fmaf(w, u.z, v.z), fmaf(w, u.w, v.w));
        }
    }
    if (b.z) {
        const float* p = b.z + (size_t)t * b.ldz + c;
#pragma unroll 4
        for (int i = 1; i < b.zparts; ++i) g = f4_add(g, load4<float>(p + i * b.zstride));
    }
}

__device__ __forceinline__ float branch1(const BranchSource& b, int t, int c, int D) {
    float v = 0.f;
    if (b.parts > 0) {
        for (int i = 0; i < b.parts; ++i) v += b.y[i * b.stride + (size_t)t * D + c];
        if (b.bias) v += b.bias[c];
    } else {
        for (int s = 0; s < b.top; ++s) {
            const int row = b.pair_row[(size_t)t * b.top + s];
            if (row >= 0) v = fmaf(b.weight[(size_t)t * b.top + s], b.y[(size_t)row * D + c], v);
        }
    }
    if (b.z) {
        float g = 0.f;
        for (int i = 0; i < b.zparts; ++i) g += b.z[i * b.zstride + (size_t)t * b.ldz + c];
        v *= sigmoid_f(g + (b.zbias ? b.zbias[c] : 0.f));
    }
    return v;
}

// One block per row; a thread owns NV float4 of it, blockDim float4 apart.  What does not change between steps (norm
// weight, biases, shift) is fetched before the wait for the previous kernel.
template <int NV, int MODE, typename O>
__global__ void __launch_bounds__(NV == 1 ? 1024 : 512)
gated_norm_add_kernel(float* __restrict__ x, const BranchSource b, const float* __restrict__ w, O* __restrict__ out,
                      int D, float eps, const ShiftAhead sa, unsigned* err) {
    __shared__ float red[32];
    pdl_launch_dependents();
    const int t = blockIdx.x;
    float4 wv[NV], bv[NV], zb[NV];
    if (NV == 1) {
        const int c = threadIdx.x * 4;
        wv[0] = bv[0] = zb[0] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < D) {
            wv[0] = load4<float>(w + c);
            if (b.bias) bv[0] = load4<float>(b.bias + c);
            if (b.zbias) zb[0] = load4<float>(b.zbias + c);
        }
    }
    pdl_wait();
    float4 v[NV], g[NV], xv[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 4;
        v[k] = g[k] = xv[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= D) continue;
        xv[k] = load4<float>(x + (size_t)t * D + c);
        branch_loads<MODE>(b, t, c, D, v[k], g[k]);
    }
    int slot = -1;
    if (sa.out) slot = sa.slots[sa.token_req[t]];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 4;
        if (c >= D) continue;
        if (NV > 1) {
            if (b.bias) bv[k] = load4<float>(b.bias + c);
            if (b.zbias) zb[k] = load4<float>(b.zbias + c);
        }
        if (b.bias) v[k] = f4_add(v[k], bv[k]);
        if (b.z) {
            if (b.zbias) g[k] = f4_add(g[k], zb[k]);
            v[k] = make_float4(v[k].x * sigmoid_f(g[k].x), v[k].y * sigmoid_f(g[k].y), v[k].z * sigmoid_f(g[k].z),
                               v[k].w * sigmoid_f(g[k].w));
        }
        ss += v[k].x * v[k].x;
        ss += v[k].y * v[k].y;
        ss += v[k].z * v[k].z;
        ss += v[k].w * v[k].w;
    }
    if (sa.out && (slot < 0 || slot >= sa.max_slots)) {
        if (threadIdx.x == 0) atomicOr(err, AIE_DEV_SLOT_OOB);
        slot = -1;
    }
    float4 old = make_float4(0.f, 0.f, 0.f, 0.f), sh = old;      // (with NV 1) the state and the shift, on their way meanwhile
    if (NV == 1 && slot >= 0 && threadIdx.x * 4 < D) {
        old = load4<float>(sa.state + (size_t)slot * D + threadIdx.x * 4);
        sh = load4<float>(sa.shift + threadIdx.x * 4);
    }
    ss = block_sum(ss, red);
    const float rinv = 1.0f / sqrtf(ss / (float)D + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 4;
        if (c >= D) continue;
        if (NV > 1) wv[k] = load4<float>(w + c);
        const float4 s = make_float4(xv[k].x + (v[k].x * rinv) * wv[k].x, xv[k].y + (v[k].y * rinv) * wv[k].y,
                                     xv[k].z + (v[k].z * rinv) * wv[k].z, xv[k].w + (v[k].w * rinv) * wv[k].w);
        store4<float>(x + (size_t)t * D + c, s);
        if (out) store4<O>(out + (size_t)t * D + c, s);
        if (slot >= 0) {
            float* st = sa.state + (size_t)slot * D + c;
            const float4 p = NV == 1 ? old : load4<float>(st), f = NV == 1 ? sh : load4<float>(sa.shift + c);
            store4<O>((O*)sa.out + (size_t)t * D + c, make_float4(shifted_f(s.x, p.x, f.x), shifted_f(s.y, p.y, f.y),
                                                                  shifted_f(s.z, p.z, f.z), shifted_f(s.w, p.w, f.w)));
            store4<float>(st, s);
        }
    }
}

// any width: the row waits in shared memory
template <typename O>
__global__ void gated_norm_add_any_kernel(float* __restrict__ x, const BranchSource b, const float* __restrict__ w,
                                          O* __restrict__ out, int D, float eps, const ShiftAhead sa, unsigned* err) {
    extern __shared__ float gn_row[];        // D + 32
    float* red = gn_row + D;
    const int t = blockIdx.x;
    float ss = 0.f;
    for (int c = threadIdx.x; c < D; c += blockDim.x) {
        const float v = branch1(b, t, c, D);
        gn_row[c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float rinv = 1.0f / sqrtf(ss / (float)D + eps);
    int slot = -1;
    if (sa.out) {
        slot = sa.slots[sa.token_req[t]];
        if (slot < 0 || slot >= sa.max_slots) {
            if (threadIdx.x == 0) atomicOr(err, AIE_DEV_SLOT_OOB);
            slot = -1;
        }
    }
    for (int c = threadIdx.x; c < D; c += blockDim.x) {
        const float s = x[(size_t)t * D + c] + (gn_row[c] * rinv) * w[c];
        x[(size_t)t * D + c] = s;
        if (out) out[(size_t)t * D + c] = from_f32<O>(s);
        if (slot >= 0) {
            float* st = sa.state + (size_t)slot * D + c;
            ((O*)sa.out)[(size_t)t * D + c] = from_f32<O>(shifted_f(s, *st, sa.shift[c]));
            *st = s;
        }
    }
}

extern "C" int aie_gated_norm_add(float* x, const float* y, int parts, long long stride, const float* bias,
                                  const int* pair_row, const float* weight, int top, const float* z, int zparts,
                                  long long zstride, int ldz, const float* zbias, const float* w, void* out, int out_dtype,
                                  int T, int D, float eps, const float* next_shift, float* next_state, void* next_out,
                                  const int* slots, const int* token_req, int max_slots, unsigned* err, cudaStream_t st) {
    if (T <= 0) return 0;
    if (D <= 0 || (parts <= 0 && (!pair_row || !weight || top <= 0)) || (z && (zparts < 1 || ldz < D)) ||
        (next_out && (!next_shift || !next_state)))
        return AIE_BAD_ARG;
    const BranchSource b = {y, (size_t)stride, parts, bias, pair_row, weight, top, z, (size_t)zstride, zparts, ldz, zbias};
    const ShiftAhead sa = {next_shift, next_state, next_out, slots, token_req, max_slots};
    const size_t al = (size_t)x | (size_t)y | (size_t)bias | (size_t)z | (size_t)zbias | (size_t)w | (size_t)out |
                      (size_t)next_shift | (size_t)next_state | (size_t)next_out;
    const bool vec = D % 4 == 0 && ldz % 4 == 0 && stride % 4 == 0 && zstride % 4 == 0 && !(al & 15);
    const int f4 = D / 4;
    const int mode = parts <= 0 ? 2 : (parts == 1 && zparts == 1 ? 1 : 0);
    // few rows: a thread a float4, so that a row's latency is one load's; many: two and more, more blocks an SM
    const int nv = f4 <= 256 || (T <= 2 * aie_sm_count() && f4 <= 1024) ? 1 : (f4 <= 1024 ? 2 : 4);
#define GO(NV, M, O)                                                                                                     \
    launch_pdl(gated_norm_add_kernel<NV, M, O>, dim3(T), dim3(((f4 + NV - 1) / NV + 31) / 32 * 32), 0, st, x, b, w,        \
               (O*)out, D, eps, sa, err)
#define GO_M(NV, O)                                                                                                      \
    if (mode == 0) GO(NV, 0, O);                                                                                         \
    else if (mode == 1) GO(NV, 1, O);                                                                                    \
    else GO(NV, 2, O)
#define GO_O(O)                                                                                                          \
    if (vec && nv == 1) {                                                                                                \
        GO_M(1, O);                                                                                                      \
    } else if (vec && nv == 2) {                                                                                         \
        GO_M(2, O);                                                                                                      \
    } else if (vec && f4 <= 2048) {                                                                                      \
        GO_M(4, O);                                                                                                      \
    } else {                                                                                                             \
        const size_t smem = (size_t)(D + 32) * sizeof(float);                                                            \
        if (smem > 200 * 1024) return AIE_UNSUPPORTED;                                                                   \
        if (smem > 48 * 1024)                                                                                            \
            cudaFuncSetAttribute(gated_norm_add_any_kernel<O>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
        gated_norm_add_any_kernel<O><<<T, 256, smem, st>>>(x, b, w, (O*)out, D, eps, sa, err);                           \
    }
    if (out_dtype == AIE_F32) {
        GO_O(float)
    } else if (out_dtype == AIE_BF16) {
        GO_O(bf16)
    } else {
        return AIE_BAD_ARG;
    }
#undef GO_O
#undef GO_M
#undef GO
    AIE_LAUNCH_CHECK();
}

// ---------------------------------------------------------------------------
// out[t, c] = gelu_tanh(sum of the parts of z[t, c]) * table[ids[t], off + c]
// ---------------------------------------------------------------------------
__device__ __forceinline__ float gelu_tanh_f(float g) {
    return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
}

// blockDim = (columns, rows of the block); VEC: four columns a thread
template <typename E, typename O, bool VEC>
__global__ void side_gate_kernel(const float* __restrict__ z, int parts, size_t stride, int ldz,
                                 const int* __restrict__ ids, const E* __restrict__ table, int vocab, int ld_table,
                                 int off, O* __restrict__ out, int T, int n, unsigned* err) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x * blockDim.y + threadIdx.y;
    if (t >= T) return;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0) atomicOr(err, AIE_DEV_TOKEN_OOB);
    const E* e = table + (size_t)(ok ? id : 0) * ld_table + off;
    const float* p = z + (size_t)t * ldz;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < n; c += blockDim.x * 4) {
            float4 w = load4<E>(e + c), g = load4<float>(p + c);
            if (!ok) w = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int i = 1; i < parts; ++i) g = f4_add(g, load4<float>(p + i * stride + c));
            store4<O>(out + (size_t)t * n + c, make_float4(gelu_tanh_f(g.x) * w.x, gelu_tanh_f(g.y) * w.y,
                                                           gelu_tanh_f(g.z) * w.z, gelu_tanh_f(g.w) * w.w));
        }
    } else {
        for (int c = threadIdx.x; c < n; c += blockDim.x) {
            float g = 0.f;
            for (int i = 0; i < parts; ++i) g += p[i * stride + c];
            out[(size_t)t * n + c] = from_f32<O>(ok ? gelu_tanh_f(g) * to_f32<E>(e[c]) : 0.f);
        }
    }
}

extern "C" int aie_side_gate(const float* z, int parts, long long stride, int ldz, const int* ids, const void* table,
                             int table_dtype, int vocab, int ld_table, int off, void* out, int out_dtype, int T, int n,
                             unsigned* err, cudaStream_t st) {
    if (T <= 0) return 0;
    if (n <= 0 || parts < 1 || ldz < n || off < 0 || off + n > ld_table) return AIE_BAD_ARG;
    const bool vec = n % 4 == 0 && ldz % 4 == 0 && stride % 4 == 0 && ld_table % 4 == 0 && off % 4 == 0 &&
                     !(((size_t)z | (size_t)table | (size_t)out) & 15);
    const int per = vec ? n / 4 : n;
    const int bx = per >= 128 ? 128 : (per + 7) / 8 * 8, by = T >= 256 && bx <= 64 ? 128 / bx : 1;
    const dim3 block(bx, by), grid((T + by - 1) / by);
#define GO(E, O)                                                                                                      \
    if (vec) launch_pdl(side_gate_kernel<E, O, true>, grid, block, 0, st, z, parts, (size_t)stride, ldz, ids,           \
                        (const E*)table, vocab, ld_table, off, (O*)out, T, n, err);                                     \
    else launch_pdl(side_gate_kernel<E, O, false>, grid, block, 0, st, z, parts, (size_t)stride, ldz, ids,              \
                    (const E*)table, vocab, ld_table, off, (O*)out, T, n, err)
    if (table_dtype == AIE_F32 && out_dtype == AIE_F32) {
        GO(float, float);
    } else if (table_dtype == AIE_BF16 && out_dtype == AIE_BF16) {
        GO(bf16, bf16);
    } else if (table_dtype == AIE_F32 && out_dtype == AIE_BF16) {
        GO(float, bf16);
    } else if (table_dtype == AIE_BF16 && out_dtype == AIE_F32) {
        GO(bf16, float);
    } else {
        return AIE_BAD_ARG;
    }
#undef GO
    AIE_LAUNCH_CHECK();
}

// ---------------------------------------------------------------------------
// a [T, H, 2, e] float32: o = a[.., 0, :] - lambda a[.., 1, :];  out [T, H e] = o / sqrt(mean(o^2) + eps) * factor.
// A warp per (token, head).
// ---------------------------------------------------------------------------
template <typename O>
__global__ void map_difference_kernel(const float* __restrict__ a, float lambda, float eps, float factor,
                                      O* __restrict__ out, long long rows, int e) {
    pdl_launch_dependents();
    pdl_wait();
    const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (row >= rows) return;
    const float* p = a + (size_t)row * 2 * e;
    float ss = 0.f;
    for (int c = lane; c < e; c += 32) {
        const float o = fmaf(-lambda, p[e + c], p[c]);
        ss += o * o;
    }
    ss = warp_sum(ss);
    const float inv = factor / sqrtf(ss / (float)e + eps);
    for (int c = lane; c < e; c += 32) out[(size_t)row * e + c] = from_f32<O>(fmaf(-lambda, p[e + c], p[c]) * inv);
}

// e a multiple of 4, at most 128: the row stays in registers, one 16-byte load per map and lane
template <typename O>
__global__ void map_difference4_kernel(const float* __restrict__ a, float lambda, float eps, float factor,
                                       O* __restrict__ out, long long rows, int e) {
    pdl_launch_dependents();
    pdl_wait();
    const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int c = (threadIdx.x & 31) * 4;
    if (row >= rows) return;
    const float* p = a + (size_t)row * 2 * e;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < e) {
        const float4 u = load4<float>(p + c), v = load4<float>(p + e + c);
        o = make_float4(fmaf(-lambda, v.x, u.x), fmaf(-lambda, v.y, u.y), fmaf(-lambda, v.z, u.z), fmaf(-lambda, v.w, u.w));
    }
    const float ss = warp_sum(o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w);
    const float inv = factor / sqrtf(ss / (float)e + eps);
    if (c < e) store4<O>(out + (size_t)row * e + c, make_float4(o.x * inv, o.y * inv, o.z * inv, o.w * inv));
}

extern "C" int aie_map_difference(const float* a, float lambda, float eps, float factor, void* out, int out_dtype,
                                  long long rows, int e, cudaStream_t st) {
    if (rows <= 0) return 0;
    if (e <= 0) return AIE_BAD_ARG;
    const bool vec = e % 4 == 0 && e <= 128;
    const dim3 grid((unsigned)((rows + 3) / 4));
#define GO(O)                                                                                                          \
    if (vec) launch_pdl(map_difference4_kernel<O>, grid, dim3(128), 0, st, a, lambda, eps, factor, (O*)out, rows, e);     \
    else launch_pdl(map_difference_kernel<O>, grid, dim3(128), 0, st, a, lambda, eps, factor, (O*)out, rows, e)
    if (out_dtype == AIE_F32) {
        GO(float);
    } else if (out_dtype == AIE_BF16) {
        GO(bf16);
    } else {
        return AIE_BAD_ARG;
    }
#undef GO
    AIE_LAUNCH_CHECK();
}

// ---------------------------------------------------------------------------
// z: logits [zparts, T, ldz] (E of each row), bias [E] or null.  A warp per token; lane l holds the logits l, l + 32, ...
// (NE of them).  Ties go to the lower index.
// ---------------------------------------------------------------------------
template <int NE>
__global__ void route_chosen_kernel(const float* __restrict__ z, int parts, size_t stride, int ldz,
                                    const float* __restrict__ bias, int T, int E, int top, int* __restrict__ ids,
                                    float* __restrict__ weights) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= T) return;
    float v[NE];
#pragma unroll
    for (int k = 0; k < NE; ++k) {
        const int e = lane + 32 * k;
        float s = -INFINITY;
        if (e < E) {
            s = 0.f;
#pragma unroll 4
            for (int p = 0; p < parts; ++p) s += z[p * stride + (size_t)t * ldz + e];
            if (bias) s += bias[e];
        }
        v[k] = s;
    }
    unsigned taken = 0u;                 // bit k: this lane's k-th logit is chosen
    float best0 = 0.f, sum = 0.f, mine = 0.f;      // lane l keeps the weight of choice l
    for (int s = 0; s < top; ++s) {
        float bv = -INFINITY;
        int be = 0x7fffffff;
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            const int e = lane + 32 * k;
            if (e < E && !(taken >> k & 1u) && (v[k] > bv || be == 0x7fffffff)) {
                bv = v[k];
                be = e;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (oe != 0x7fffffff && (be == 0x7fffffff || ov > bv || (ov == bv && oe < be))) {
                bv = ov;
                be = oe;
            }
        }
        if ((be & 31) == lane) taken |= 1u << (be >> 5);
        if (s == 0) best0 = bv;
        const float w = expf(bv - best0);
        sum += w;
        if (lane == 0) ids[(size_t)t * top + s] = be;
        if ((s & 31) == lane) {
            if (s >= 32) weights[(size_t)t * top + s] = w;       // more than 32 choices: finished below
            else mine = w;
        }
    }
    if (lane < top) weights[(size_t)t * top + lane] = mine / sum;
    for (int s = lane + 32; s < top; s += 32) weights[(size_t)t * top + s] /= sum;
}

extern "C" int aie_route_chosen(const float* z, int parts, long long stride, int ldz, const float* bias, int T, int E,
                                int top, int* ids, float* weights, cudaStream_t st) {
    if (T <= 0) return 0;
    if (E <= 0 || top <= 0 || top > E || ldz < E || parts < 1) return AIE_BAD_ARG;
    if (E > 1024) return AIE_UNSUPPORTED;
    const dim3 grid((T + 3) / 4);
#define GO(NE) launch_pdl(route_chosen_kernel<NE>, grid, dim3(128), 0, st, z, parts, (size_t)stride, ldz, bias, T, E, top, ids, weights)
    if (E <= 32) GO(1);
    else if (E <= 64) GO(2);
    else if (E <= 128) GO(4);
    else if (E <= 256) GO(8);
    else GO(32);
#undef GO
    AIE_LAUNCH_CHECK();
}
