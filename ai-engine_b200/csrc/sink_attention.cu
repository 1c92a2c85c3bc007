// Softmax attention with a distance bias, a window that keeps the first tokens, a sink and a gate per head,
// over a paged cache of one plane whose rows hold a key (d elements) and behind it a value (e elements).
//
//   s(i, j) = (q_i . k_j) * scale * temp[h] - slope[h] * (i - j)
//   i reads j  iff  j <= i and (window <= 0 or i - j < window or j < keep_first)
//   out_i = gate[i, h] * sum_j exp(s(i, j)) v_j / (exp(sink[h]) + sum_j exp(s(i, j)))
//
// cap > 0: (q_i . k_j) * scale * temp[h] is replaced by cap * tanh(it / cap).  gate_logits: every output element is
// multiplied by the sigmoid of a logit of its own.  tied: values are the keys, and a row is that one vector of d == e.
// The sink is a term of the denominator that has no key and no value.  Scores, weights and sums are float32.
// chunk > 0 (without a window): i reads j  iff  j <= i and j / chunk == i / chunk.
// maps > 1: a key/value head has `maps` keys in front of its one value, a row is [k_0 .. k_(maps-1) | v]; query head h
// of the H (all maps counted) reads key h % maps of key/value head h / (H / G).
//
//   sink_attn_prepare    from a step's fused projection [q | k | v | gate logits] (float32): adds the biases,
//                        writes q in the compute dtype, divides each head's value by its root mean square
//                        (no weight) and writes key and value into the token's cache row, gate = sigmoid.
//   normed_attn_prepare  for a layer that norms and rotates instead: from a fused projection whose first columns are
//                        [q | k | v] it adds the biases, divides all of q (and all of k) by its root mean square
//                        over the whole projection, times a weight per element, rotates the first rot_dims
//                        elements of every head (neighbouring pairs, or halves), mixes the value with another
//                        layer's value of the same token, and writes q and the cache row [k | v].  With
//                        `per_head` every head (and map) of q and k is normed by itself, with one weight of d
//                        elements for all of them; with `unit` every head is divided by its root mean square behind
//                        the rotation, without a weight.
//   sink_attention_plain one block per (query token, head), any sizes up to 256; keys are walked in chunks of
//                        128 that start at multiples of 128 of the absolute key position, so the order of
//                        every addition depends on the query's position only.
#include "common.cuh"

#define SA_CHUNK 128

template <typename A, typename C>
__global__ void __launch_bounds__(256)
sink_attn_prepare_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ bias, A* __restrict__ q_out,
                         C* __restrict__ pages, float* __restrict__ gate_out, const int* __restrict__ positions,
                         const int* __restrict__ token_req, const int* __restrict__ block_table, int bt_width,
                         int num_pages, int P, int H, int G, int d, int e, float eps, int write, unsigned* err) {
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const float* row = proj + (size_t)t * ld;
    const int nq = H * d, nk = G * d, nv = G * e;
    for (int c = tid; c < nq; c += blockDim.x)
        q_out[(size_t)t * nq + c] = from_f32<A>(row[c] + (bias ? bias[c] : 0.f));
    for (int h = tid; h < H; h += blockDim.x)
        gate_out[(size_t)t * H + h] = 1.f / (1.f + expf(-row[nq + nk + nv + h]));
    if (!write) return;
    const int pos = positions[t], r = token_req[t];
    const int pidx = pos / P;
    const int page = pidx < bt_width ? block_table[(size_t)r * bt_width + pidx] : -1;
    if (page < 0 || page >= num_pages) {
        if (tid == 0) atomicOr(err, AIE_DEV_PAGE_OOB);
        return;
    }
    const int w = d + e;
    for (int g = warp; g < G; g += nw) {          // a warp per key/value head
        C* dst = pages + (((size_t)page * G + g) * P + (pos % P)) * w;
        for (int c = lane; c < d; c += 32)
            dst[c] = from_f32<C>(row[nq + g * d + c] + (bias ? bias[nq + g * d + c] : 0.f));
        float ss = 0.f;
        for (int c = lane; c < e; c += 32) {
            const float v = row[nq + nk + g * e + c] + (bias ? bias[nq + nk + g * e + c] : 0.f);
            ss += v * v;
        }
        ss = warp_sum(ss);
        const float inv = rsqrtf(ss / (float)e + eps);
        for (int c = lane; c < e; c += 32) {
            const float v = row[nq + nk + g * e + c] + (bias ? bias[nq + nk + g * e + c] : 0.f);
            dst[d + c] = from_f32<C>(v * inv);
        }
    }
}

extern "C" int aie_sink_attn_prepare(const float* proj, int ld, const float* bias, void* q_out, int q_dtype, void* pages,
                                     int cache_dtype, float* gate_out, const int* positions, const int* token_req,
                                     const int* block_table, int bt_width, int num_pages, int P, int T, int H, int G,
                                     int d, int e, float eps, int write, unsigned* err, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || e <= 0 || q_dtype != cache_dtype) return AIE_BAD_ARG;
#define AIE_SAP(A)                                                                                                    \
    sink_attn_prepare_kernel<A, A><<<T, 256, 0, stream>>>(proj, ld, bias, (A*)q_out, (A*)pages, gate_out, positions,    \
                                                         token_req, block_table, bt_width, num_pages, P, H, G, d, e,  \
                                                         eps, write, err)
    if (q_dtype == AIE_F32) AIE_SAP(float);
    else if (q_dtype == AIE_BF16) AIE_SAP(bf16);
    else return AIE_BAD_ARG;
#undef AIE_SAP
    AIE_LAUNCH_CHECK();
}

// The two elements of pair j (of rot_dims / 2) of a head that starts at x, turned by `pos`: neighbours (2j, 2j + 1) or,
// with `halves`, (j, j + rot_dims / 2).  One sincosf a pair.
__device__ __forceinline__ void head_pair_rotated(const float* x, int j, int rot_dims, int halves, int pos,
                                                  const float* __restrict__ inv_freq, int* ia, int* ib, float* ya,
                                                  float* yb) {
    const int a = halves ? j : 2 * j, b = halves ? j + (rot_dims >> 1) : 2 * j + 1;
    float sn, cs;
    sincosf((float)pos * inv_freq[j], &sn, &cs);
    *ia = a;
    *ib = b;
    *ya = x[a] * cs - x[b] * sn;
    *yb = x[b] * cs + x[a] * sn;
}

// proj [T, >= H d + G d + G e] float32; bias [H d + G d + G e] or null; q_w [H d], k_w [G d] float32 or null (no norm).
// mix_from [T, G e] float32 with lambda (one float on the device): v <- (1 - lambda) v + lambda mix_from[t].
// v_keep [T, G e]: receives v as it is cached, in float32 (for the layers that mix with it).
template <typename A>
__global__ void __launch_bounds__(256)
normed_attn_prepare_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ bias,
                           const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                           const float* __restrict__ inv_freq, int rot_dims, int halves,
                           const float* __restrict__ mix_from, const float* __restrict__ lambda,
                           float* __restrict__ v_keep, A* __restrict__ q_out, A* __restrict__ pages,
                           const int* __restrict__ positions, const int* __restrict__ token_req,
                           const int* __restrict__ block_table, int bt_width, int num_pages, int P, int H, int G, int d,
                           int e, int maps, int per_head, int write, unsigned* err) {
    extern __shared__ __align__(16) float np_sm[];     // q (H d) | k (G maps d) | 32
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x;
    const int K = G * maps;                             // keys of a token
    const int nq = H * d, nk = K * d, nv = G * e;
    float* qs = np_sm;
    float* ks = qs + nq;
    float* red = ks + nk;
    const float* row = proj + (size_t)t * ld;
    float ssq = 0.f, ssk = 0.f;
    for (int c = tid; c < nq; c += blockDim.x) {
        const float x = row[c] + (bias ? bias[c] : 0.f);
        qs[c] = x;
        ssq += x * x;
    }
    for (int c = tid; c < nk; c += blockDim.x) {
        const float x = row[nq + c] + (bias ? bias[nq + c] : 0.f);
        ks[c] = x;
        ssk += x * x;
    }
    if (q_w && per_head) {                              // a warp per head
        __syncthreads();
        for (int hh = tid >> 5; hh < H + K; hh += blockDim.x >> 5) {
            float* x = hh < H ? qs + hh * d : ks + (hh - H) * d;
            const float* wv = hh < H ? q_w : k_w;
            float ss = 0.f;
            for (int c = tid & 31; c < d; c += 32) ss += x[c] * x[c];
            ss = warp_sum(ss);
            const float inv = 1.0f / sqrtf(ss / (float)d + eps);
            for (int c = tid & 31; c < d; c += 32) x[c] = (x[c] * inv) * wv[c];
        }
    } else if (q_w) {
        ssq = block_sum(ssq, red);
        ssk = block_sum(ssk, red);
        const float rq = 1.0f / sqrtf(ssq / (float)nq + eps), rk = 1.0f / sqrtf(ssk / (float)nk + eps);
        for (int c = tid; c < nq; c += blockDim.x) qs[c] = (qs[c] * rq) * q_w[c];
        for (int c = tid; c < nk; c += blockDim.x) ks[c] = (ks[c] * rk) * k_w[c];
    }
    __syncthreads();
    const int pos = positions[t];
    const int half = rot_dims >> 1, rest = d - rot_dims;
    for (int p = tid; p < H * half; p += blockDim.x) {            // a thread a pair
        const int hh = p / half, j = p - hh * half;
        int ia, ib;
        float ya, yb;
        head_pair_rotated(qs + hh * d, j, rot_dims, halves, pos, inv_freq, &ia, &ib, &ya, &yb);
        q_out[(size_t)t * nq + hh * d + ia] = from_f32<A>(ya);
        q_out[(size_t)t * nq + hh * d + ib] = from_f32<A>(yb);
    }
    for (int p = tid; p < H * rest; p += blockDim.x) {            // what the rotation leaves as it is
        const int c = (p / rest) * d + rot_dims + p % rest;
        q_out[(size_t)t * nq + c] = from_f32<A>(qs[c]);
    }
    const int pidx = pos / P;
    const int page = (pos >= 0 && pidx < bt_width) ? block_table[(size_t)token_req[t] * bt_width + pidx] : -1;
    const bool page_ok = page >= 0 && page < num_pages;
    if (write && !page_ok && tid == 0) atomicOr(err, AIE_DEV_PAGE_OOB);
    const int w = maps * d + e;
    A* base = pages + ((size_t)(page_ok ? page : 0) * G * P + (pos % P)) * w;
    if (write && page_ok) {
        for (int p = tid; p < K * half; p += blockDim.x) {
            const int k = p / half, j = p - k * half;
            int ia, ib;
            float ya, yb;
            head_pair_rotated(ks + k * d, j, rot_dims, halves, pos, inv_freq, &ia, &ib, &ya, &yb);
            A* dst = base + (size_t)(k / maps) * P * w + (k % maps) * d;
            dst[ia] = from_f32<A>(ya);
            dst[ib] = from_f32<A>(yb);
        }
        for (int p = tid; p < K * rest; p += blockDim.x) {
            const int k = p / rest, i = rot_dims + p % rest;
            base[(size_t)(k / maps) * P * w + (k % maps) * d + i] = from_f32<A>(ks[k * d + i]);
        }
    }
    const float lam = mix_from ? lambda[0] : 0.f;
    for (int c = tid; c < nv; c += blockDim.x) {
        float v = row[nq + nk + c] + (bias ? bias[nq + nk + c] : 0.f);
        if (mix_from) v = (1.0f - lam) * v + lam * mix_from[(size_t)t * nv + c];
        if (v_keep) v_keep[(size_t)t * nv + c] = v;
        if (write && page_ok) {
            const int g = c / e;
            base[(size_t)g * P * w + maps * d + (c - g * e)] = from_f32<A>(v);
        }
    }
}

// The same for heads that are normed one by one (or not), rotated in neighbouring pairs (or not) and not mixed: a warp
// per head of q, k or v, a head's elements in registers (d <= 256).  A norm with weights comes ahead of the rotation,
// `unit` behind it; rotated elements are multiplied by `mag`.
template <typename A>
__global__ void __launch_bounds__(256)
head_normed_prepare_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ bias,
                           const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                           const float* __restrict__ inv_freq, int rot_dims, float mag, int unit, A* __restrict__ q_out,
                           A* __restrict__ pages, const int* __restrict__ positions, const int* __restrict__ token_req,
                           const int* __restrict__ block_table, int bt_width, int num_pages, int P, int H, int G, int d,
                           int e, int maps, int tied, int write, unsigned* err) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31;
    const int K = G * maps, nq = H * d, nk = K * d;
    const int hh = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);      // heads of q, then of k, then of v
    if (hh >= H + K + (tied ? 0 : G) || (hh >= H && !write)) return;
    const bool is_v = hh >= H + K;
    const int n = is_v ? e : d;
    const int at = is_v ? nq + nk + (hh - H - K) * e : hh * d;
    const float* row = proj + (size_t)t * ld + at;
    const float* b = bias ? bias + at : nullptr;
    A* dst = q_out + (size_t)t * nq + hh * d;
    if (hh >= H) {
        const int pos = positions[t], pidx = pos / P;
        const int page = (pos >= 0 && pidx < bt_width) ? block_table[(size_t)token_req[t] * bt_width + pidx] : -1;
        if (page < 0 || page >= num_pages) {
            if (lane == 0) atomicOr(err, AIE_DEV_PAGE_OOB);
            return;
        }
        const int k = hh - H, g = is_v ? k - K : k / maps;
        dst = pages + (((size_t)page * G + g) * P + (pos - pidx * P)) * (maps * d + (tied ? 0 : e)) + (is_v ? maps * d : (k % maps) * d);
    }
    float x[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        x[i] = c < n ? row[c] + (b ? b[c] : 0.f) : 0.f;
        ss += x[i] * x[i];
    }
    const float* w = is_v ? nullptr : (hh < H ? q_w : k_w);
    if (w) {
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)d + eps);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = lane + 32 * i;
            if (c < n) x[i] = (x[i] * inv) * w[c];
        }
    }
    if (rot_dims > 0 && !is_v) {                        // the other element of a pair is the neighbouring lane's
        const float pos = (float)positions[t];
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = lane + 32 * i;
            const float other = __shfl_xor_sync(0xffffffffu, x[i], 1);
            if (c < rot_dims) {
                float sn, cs;
                sincosf(pos * inv_freq[c >> 1], &sn, &cs);
                sn *= mag;
                cs *= mag;
                x[i] = (c & 1) ? x[i] * cs + other * sn : x[i] * cs - other * sn;
            }
            ss += x[i] * x[i];
        }
    }
    if (unit && !is_v) {
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)d + eps);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] *= inv;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c < n) dst[c] = from_f32<A>(x[i]);
    }
}

// The same for sizes in steps of 4 (d <= 128): groups of L lanes (a power of two, L >= d / 4) hold a head of q or k,
// four elements (two pairs) a lane; the last blocks copy the values.  A block makes a token's angles once, in shared
// memory (rot_dims <= 128).
template <typename A>
__global__ void __launch_bounds__(256)
head_normed_prepare4_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ bias,
                            const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                            const float* __restrict__ inv_freq, int rot_dims, float mag, int unit, A* __restrict__ q_out,
                            A* __restrict__ pages, const int* __restrict__ positions, const int* __restrict__ token_req,
                            const int* __restrict__ block_table, int bt_width, int num_pages, int P, int H, int G, int d,
                            int e, int maps, int L, int head_blocks, int tied, int write, unsigned* err) {
    __shared__ float2 turn[64];                          // (cos, sin) of the token's angles, times mag
    pdl_launch_dependents();
    if (rot_dims > 0 && blockIdx.y < head_blocks) {      // positions and frequencies are no kernel's output
        for (int j = threadIdx.x; j < rot_dims / 2; j += blockDim.x) {
            float sn, cs;
            sincosf((float)positions[blockIdx.x] * inv_freq[j], &sn, &cs);
            turn[j] = make_float2(cs * mag, sn * mag);
        }
        __syncthreads();
    }
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31;
    const int K = G * maps, nq = H * d, nk = K * d, w_row = maps * d + (tied ? 0 : e);
    const float* row = proj + (size_t)t * ld;
    A* base = nullptr;                                   // the token's place in the page, of key/value head 0
    const bool values = blockIdx.y >= head_blocks;
    const int per = 32 / L;
    const int hh = (blockIdx.y * 8 + (threadIdx.x >> 5)) * per + lane / L, c = (lane & (L - 1)) * 4;
    if (values || hh >= H) {
        const int pos = positions[t], pidx = pos / P;
        const int page = (pos >= 0 && pidx < bt_width) ? block_table[(size_t)token_req[t] * bt_width + pidx] : -1;
        if (page >= 0 && page < num_pages) base = pages + ((size_t)page * G * P + (pos - pidx * P)) * w_row;
        else if (write && (threadIdx.x & 31) == 0) atomicOr(err, AIE_DEV_PAGE_OOB);
    }
    if (values) {
        const int i = ((blockIdx.y - head_blocks) * blockDim.x + threadIdx.x) * 4;
        if (i >= G * e || !base || !write) return;
        float4 v = load4<float>(row + nq + nk + i);
        if (bias) {
            const float4 b = load4<float>(bias + nq + nk + i);
            v = make_float4(v.x + b.x, v.y + b.y, v.z + b.z, v.w + b.w);
        }
        const int g = i / e;
        store4<A>(base + (size_t)g * P * w_row + maps * d + (i - g * e), v);
        return;
    }
    const bool on = hh < H + K && c < d;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f), w = x;
    if (on) {
        x = load4<float>(row + hh * d + c);
        if (bias) {
            const float4 b = load4<float>(bias + hh * d + c);
            x = make_float4(x.x + b.x, x.y + b.y, x.z + b.z, x.w + b.w);
        }
        if (q_w) w = load4<float>((hh < H ? q_w : k_w) + c);
    }
    if (q_w) {
        float ss = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
        for (int o = L >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.0f / sqrtf(ss / (float)d + eps);
        x = make_float4((x.x * inv) * w.x, (x.y * inv) * w.y, (x.z * inv) * w.z, (x.w * inv) * w.w);
    }
    if (on && c < rot_dims) {
        const float2 a = turn[c >> 1];
        const float u = x.x, v = x.y;
        x.x = u * a.x - v * a.y;
        x.y = v * a.x + u * a.y;
        if (c + 2 < rot_dims) {
            const float2 b = turn[(c >> 1) + 1];
            const float u2 = x.z, v2 = x.w;
            x.z = u2 * b.x - v2 * b.y;
            x.w = v2 * b.x + u2 * b.y;
        }
    }
    if (unit) {
        float ss = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
        for (int o = L >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.0f / sqrtf(ss / (float)d + eps);
        x = make_float4(x.x * inv, x.y * inv, x.z * inv, x.w * inv);
    }
    if (!on) return;
    if (hh < H) {
        store4<A>(q_out + (size_t)t * nq + hh * d + c, x);
    } else if (base && write) {
        const int k = hh - H;
        store4<A>(base + (size_t)(k / maps) * P * w_row + (k % maps) * d + c, x);
    }
}

extern "C" int aie_normed_attn_prepare(const float* proj, int ld, const float* bias, const float* q_w, const float* k_w,
                                       float eps, const float* inv_freq, int rot_dims, int halves, float mag, int unit,
                                       int tied, const float* mix_from, const float* lambda, float* v_keep,
                                       void* q_out, void* pages, int dtype, const int* positions, const int* token_req, const int* block_table, int bt_width,
                                       int num_pages, int P, int T, int H, int G, int d, int e, int maps, int per_head,
                                       int write, unsigned* err, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (maps < 1 || H % maps || (H / maps) % G) return AIE_BAD_ARG;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || e <= 0 || rot_dims < 0 || rot_dims > d || rot_dims % 2 ||
        (mix_from && !lambda) || (q_w && !k_w) || (rot_dims > 0 && !inv_freq))
        return AIE_BAD_ARG;
    if (tied && (d != e || maps != 1)) return AIE_BAD_ARG;
    if ((per_head || !q_w) && (rot_dims == 0 || !halves) && !mix_from && !v_keep && d <= 256 && e <= 256) {
        const size_t al = (size_t)proj | (size_t)bias | (size_t)q_w | (size_t)k_w | (size_t)q_out | (size_t)pages;
        if (d % 4 == 0 && e % 4 == 0 && ld % 4 == 0 && d <= 128 && !(al & 15) && (dtype == AIE_F32 || dtype == AIE_BF16)) {
            int L = 1;
            while (L * 4 < d) L *= 2;
            const int hb = (H + G * maps + 8 * (32 / L) - 1) / (8 * (32 / L)), vb = tied ? 0 : (G * e / 4 + 255) / 256;
            const dim3 grid4(T, hb + vb);
            if (dtype == AIE_F32)
                launch_pdl(head_normed_prepare4_kernel<float>, grid4, dim3(256), 0, stream, proj, ld, bias, q_w, k_w, eps, inv_freq, rot_dims, mag, unit, (float*)q_out, (float*)pages, positions, token_req, block_table, bt_width, num_pages, P, H, G, d, e, maps, L, hb, tied, write, err);
            else
                launch_pdl(head_normed_prepare4_kernel<bf16>, grid4, dim3(256), 0, stream, proj, ld, bias, q_w, k_w, eps, inv_freq, rot_dims, mag, unit, (bf16*)q_out, (bf16*)pages, positions, token_req, block_table, bt_width, num_pages, P, H, G, d, e, maps, L, hb, tied, write, err);
            AIE_LAUNCH_CHECK();
        }
        const dim3 grid(T, (H + G * maps + G + 7) / 8);
        if (dtype == AIE_F32)
            launch_pdl(head_normed_prepare_kernel<float>, grid, dim3(256), 0, stream, proj, ld, bias, q_w, k_w, eps, inv_freq, rot_dims, mag, unit, (float*)q_out, (float*)pages, positions, token_req, block_table, bt_width, num_pages, P, H, G, d, e, maps, tied, write, err);
        else if (dtype == AIE_BF16)
            launch_pdl(head_normed_prepare_kernel<bf16>, grid, dim3(256), 0, stream, proj, ld, bias, q_w, k_w, eps, inv_freq, rot_dims, mag, unit, (bf16*)q_out, (bf16*)pages, positions, token_req, block_table, bt_width, num_pages, P, H, G, d, e, maps, tied, write, err);
        else
            return AIE_BAD_ARG;
        AIE_LAUNCH_CHECK();
    }
    if (mag != 1.f || unit || tied) return AIE_UNSUPPORTED;
    const size_t smem = ((size_t)(H + G * maps) * d + 32) * sizeof(float);
    if (smem > 200 * 1024) return AIE_UNSUPPORTED;
#define AIE_NAP(A)                                                                                                    \
    if (smem > 48 * 1024)                                                                                             \
        cudaFuncSetAttribute(normed_attn_prepare_kernel<A>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
    launch_pdl(normed_attn_prepare_kernel<A>, dim3(T), dim3(256), smem, stream, proj, ld, bias, q_w, k_w, eps, inv_freq, rot_dims, halves, \
                                                           mix_from, lambda, v_keep, (A*)q_out, (A*)pages, positions, \
                                                           token_req, block_table, bt_width, num_pages, P, H, G, d, e, \
                                                           maps, per_head, write, err)
    if (dtype == AIE_F32) {
        AIE_NAP(float);
    } else if (dtype == AIE_BF16) {
        AIE_NAP(bf16);
    } else {
        return AIE_BAD_ARG;
    }
#undef AIE_NAP
    AIE_LAUNCH_CHECK();
}

template <typename A, typename C, typename O>
__global__ void __launch_bounds__(SA_CHUNK)
sink_attention_plain_kernel(const A* __restrict__ q, const C* __restrict__ pages, O* __restrict__ out,
                            const float* __restrict__ gate, const float* __restrict__ temp,
                            const float* __restrict__ slope, const float* __restrict__ sink,
                            const int* __restrict__ positions, const int* __restrict__ token_req,
                            const int* __restrict__ block_table, int bt_width, int num_pages, int P, int H, int G,
                            int d, int e, int window, int keep_first, int chunk, int maps, float scale, float cap,
                            int tied, const float* __restrict__ gate_logits, int ld_gate,
                            const int* __restrict__ token_list, unsigned* err) {
    extern __shared__ __align__(16) float sm[];
    float* q_s = sm;                                  // d (rounded up to even)
    float* p_s = q_s + ((d + 1) & ~1);                // CHUNK
    float* red = p_s + SA_CHUNK;                      // 32
    long long* off_s = (long long*)(red + 32);        // CHUNK

    const int t = token_list ? token_list[blockIdx.x] : blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int pos = positions[t];
    const int row = token_req[t];
    const int g = h / (H / G);
    const int w = maps * d + (tied ? 0 : e), k_off = (h % maps) * d, v_off = tied ? 0 : maps * d;
    const float qs = scale * (temp ? temp[h] : 1.f), sl = slope ? slope[h] : 0.f;
    for (int c = tid; c < d; c += blockDim.x) q_s[c] = to_f32<A>(q[((size_t)t * H + h) * d + c]);
    __syncthreads();

    int lo = 0;
    if (window > 0 && pos - window + 1 > 0) lo = pos - window + 1;
    if (chunk > 0) lo = pos / chunk * chunk;
    const int kept = min(keep_first, lo);              // keys [0, kept) are read although the window has passed them
    // the sink opens the running softmax: a weight exp(sink - m) = 1 at m = sink, with no value
    float m = sink ? sink[h] : -INFINITY, l = sink ? 1.f : 0.f;
    float acc0 = 0.f, acc1 = 0.f;                      // value elements tid and tid + 128 (e <= 256)

    const int first_b = (lo / SA_CHUNK) * SA_CHUNK;    // chunk of the window's first key
    for (int c0 = 0; c0 <= pos; c0 += SA_CHUNK) {
        if (c0 >= kept && c0 < first_b) {              // between the kept keys and the window: nothing to read
            c0 = first_b - SA_CHUNK;
            continue;
        }
        const int kp = c0 + tid;
        const bool valid = kp <= pos && (kp >= lo || kp < kept);
        float s = -INFINITY;
        long long off = -1;
        if (valid) {
            const int pidx = kp / P;
            const int page = pidx < bt_width ? block_table[(size_t)row * bt_width + pidx] : -1;
            if (page < 0 || page >= num_pages) {
                atomicOr(err, AIE_DEV_PAGE_OOB);
            } else {
                off = (((long long)page * G + g) * P + (kp % P)) * w;
                const C* kr = pages + off + k_off;
                float dot = 0.f;
                for (int c = 0; c < d; ++c) dot += q_s[c] * to_f32<C>(kr[c]);
                s = dot * qs;
                if (cap > 0.f) s = cap * tanhf(s / cap);
                s -= sl * (float)(pos - kp);
            }
        }
        off_s[tid] = off;
        const float cmax = block_max(s, red);
        const float m_new = fmaxf(m, cmax);
        const float p = (off >= 0) ? expf(s - m_new) : 0.f;
        const float corr = (m == -INFINITY) ? 0.f : expf(m - m_new);
        p_s[tid] = p;
        const float csum = block_sum(p, red);          // has __syncthreads inside: p_s, off_s visible
        l = l * corr + csum;
        m = m_new;
        acc0 *= corr;
        acc1 *= corr;
        const int n = min(SA_CHUNK, pos - c0 + 1);
        for (int j = 0; j < n; ++j) {
            const long long o = off_s[j];
            if (o < 0) continue;
            const float pj = p_s[j];
            if (tid < e) acc0 += pj * to_f32<C>(pages[o + v_off + tid]);
            if (tid + SA_CHUNK < e) acc1 += pj * to_f32<C>(pages[o + v_off + tid + SA_CHUNK]);
        }
        __syncthreads();
    }
    const float inv = (l > 0.f ? 1.0f / l : 0.f) * (gate ? gate[(size_t)t * H + h] : 1.f);
    O* o = out + ((size_t)t * H + h) * e;
    const float* gl = gate_logits ? gate_logits + (size_t)t * ld_gate + (size_t)h * e : nullptr;
    if (tid < e) o[tid] = from_f32<O>(acc0 * inv * (gl ? 1.f / (1.f + expf(-gl[tid])) : 1.f));
    if (tid + SA_CHUNK < e)
        o[tid + SA_CHUNK] = from_f32<O>(acc1 * inv * (gl ? 1.f / (1.f + expf(-gl[tid + SA_CHUNK])) : 1.f));
}

extern "C" int aie_sink_attention_plain(const void* q, const void* pages, void* out, int dtype, int out_dtype, const float* gate,
                                        const float* temp, const float* slope, const float* sink, const int* positions,
                                        const int* token_req, const int* block_table, int bt_width, int num_pages,
                                        int P, int T, int H, int G, int d, int e, int window, int keep_first,
                                        int chunk, int maps, float scale, float cap, int tied, const float* gate_logits,
                                        int ld_gate, const int* token_list, unsigned* err, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (tied && (d != e || maps != 1)) return AIE_BAD_ARG;
    if (d <= 0 || d > 2 * SA_CHUNK || e <= 0 || e > 2 * SA_CHUNK || G <= 0 || H % G || H > 65535) return AIE_UNSUPPORTED;
    if (maps < 1 || (H / G) % maps || chunk < 0 || (chunk > 0 && (window > 0 || keep_first > 0))) return AIE_BAD_ARG;
    const size_t smem = (size_t)(((d + 1) & ~1) + SA_CHUNK + 32) * sizeof(float) + SA_CHUNK * sizeof(long long);
    dim3 grid(T, H);
#define AIE_SA(A, O)                                                                                                   \
    sink_attention_plain_kernel<A, A, O><<<grid, SA_CHUNK, smem, stream>>>(                                            \
        (const A*)q, (const A*)pages, (O*)out, gate, temp, slope, sink, positions, token_req, block_table, bt_width,   \
        num_pages, P, H, G, d, e, window, keep_first, chunk, maps, scale, cap, tied, gate_logits, ld_gate, token_list, err)
    if (dtype == AIE_F32 && out_dtype == AIE_F32) AIE_SA(float, float);
    else if (dtype == AIE_BF16 && out_dtype == AIE_BF16) AIE_SA(bf16, bf16);
    else if (dtype == AIE_BF16 && out_dtype == AIE_F32) AIE_SA(bf16, float);
    else return AIE_BAD_ARG;
#undef AIE_SA
    AIE_LAUNCH_CHECK();
}
