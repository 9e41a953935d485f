// Attention without a softmax for decode steps (attention_sigmoid.cu has the formulas): one new token a sequence against the
// paged cache, bfloat16.
//
// The heads' weights are mixed per key, so a CTA takes a run of a row's keys for all heads. A row's keys are dealt to
// `n_parts` CTAs in runs of whole stages; a CTA walks its run in stages of KP keys of every kv head, keys and values, which
// TMA brings through a ring of stages (128-byte swizzle, a box of KP rows x 64 columns at a time):
//   scores    keys are the 16 rows and a group's query heads the columns of a warp-level tensor-core tile, float32 sums; the
//             lanes that hold them make the weights, float32, into shared memory
//   values    a tile of 16 value columns x the group's heads, summed over the keys on the tensor cores. A lane mixes the
//             weights of the keys and the head its fragment holds (heads multiply-adds each, float32) and splits them into
//             three bfloat16 parts that hold their 24 bits
// A warp's time is the instructions it waits for one after the other, so two teams of eight warps take a run's stages in turns,
// each with weights and barriers of its own, and add their sums at the end.
// Since nothing is normalized over the keys, a CTA's sums are its part of the output; attention_sigmoid_fold adds the
// parts of a row in order. How a row is cut depends on its own position and on n_parts.
#define ABK_DEFINE_ERROR
#include "common.cuh"
#include "attention_sigmoid.cuh"
#include "mma_tiles.cuh"
#include "tc_common.cuh"
#include "tensor_map.cuh"

#define SD_WARPS 8                     // a team
#define SD_TEAM_THREADS (32 * SD_WARPS)
#define SD_MAX_STAGES 4

struct SigmoidDecode {
    const __nv_bfloat16 *q;  // row t, head h at q + t * q_row + h * head_dim
    long long q_row;
    float *parts;            // [tokens][n_parts][n_heads * v_dim]
    __nv_bfloat16 *out;      // [tokens][n_heads * v_dim]
    int n_heads, n_kv_heads, head_dim, v_dim;
    float scale, softcap;
    const float *slopes, *shift, *mix;
    const int *token_seq, *token_pos, *seq_slot;
    PagedCache cache;
    int n_parts, kp, stages;
    int *status;
};

// Keys of a CTA's run: whole stages, at least two of them, so that n_parts runs cover the row.
__host__ __device__ inline int sd_span(int keys, int n_parts, int kp) {
    const int stages = (keys + kp - 1) / kp, each = (stages + n_parts - 1) / n_parts;
    return (each < 2 ? 2 : each) * kp;
}

// The parts of shared memory behind the ring of stages (bytes).
struct SigmoidDecodeSmem {
    int k_boxes, v_boxes, stage, pitch_q, pitch_w, rows_w, pitch_m, q, w, mix, head, total;
    __host__ __device__ SigmoidDecodeSmem(int H, int G, int D, int VD, int kp, int stages) {
        k_boxes = (D + 63) / 64, v_boxes = (VD + 63) / 64;
        stage = G * (k_boxes + v_boxes) * kp * 128;
        pitch_q = (D + 15) / 16 * 16 + 8;  // elements of a query head's row
        pitch_w = kp + 8;                  // floats of a head's weights
        rows_w = (H + 3) & ~3, pitch_m = rows_w + 4;
        q = H * pitch_q * 2, w = rows_w * pitch_w * 4, mix = H * pitch_m * 4, head = H * (int)sizeof(SigmoidHead);  // (w: a buffer)
        total = 1024 + stages * stage + q + 2 * w + mix + head + 64;
        const int sums = 1024 + SD_WARPS * 16 * 512;  // the second team's, at the end, from the ring's start
        if (total < sums) total = sums;
    }
};

// Waits until stage st is asked for; false if that took longer than the library's limit.
__device__ __forceinline__ bool sd_asked(const volatile int *asked, int st) {
    if (*asked < st) {
        const uint64_t start = tc::global_ns(), limit = tc::abk_wait_limit_ns;
        while (*asked < st)
            if (tc::global_ns() - start > limit) return false;
    }
    __threadfence_block();
    return true;
}

// UNITS: tiles of 16 value columns a warp sums; NT: tiles of 8 heads a group has. ONE: eight kv heads of UNITS tiles each, so that
// a warp's tiles are one head's.
template <int UNITS, int NT, bool ONE, int TEAMS> __global__ void __launch_bounds__(SD_TEAM_THREADS * TEAMS) attention_sigmoid_decode_kernel(const __grid_constant__ CUtensorMap map_k,
                                                                                                        const __grid_constant__ CUtensorMap map_v,
                                                                                                        SigmoidDecode p) {
    extern __shared__ uint8_t sd_raw[];
    uint8_t *ring = (uint8_t *)(((uintptr_t)sd_raw + 1023) & ~(uintptr_t)1023);
    const int H = p.n_heads, G = p.n_kv_heads, D = p.head_dim, VD = p.v_dim, R = H / G, kp = p.kp;
    const SigmoidDecodeSmem sm(H, G, D, VD, kp, p.stages);
    __nv_bfloat16 *q_s = (__nv_bfloat16 *)(ring + p.stages * sm.stage);
    float *const a_s = (float *)((uint8_t *)q_s + sm.q), *const mix_s = a_s + 2 * sm.w / 4;
    SigmoidHead *const head_s = (SigmoidHead *)((uint8_t *)mix_s + sm.mix);
    __shared__ uint64_t full[SD_MAX_STAGES];
    // the last stage that was asked for into each place of the ring. A place's stages may belong to either team, and a barrier's
    // parity alone does not tell a phase from the one after next: a team waits on a barrier only once its own stage is asked for
    // (which is after the place's stage before had come and was read).
    __shared__ volatile int asked[SD_MAX_STAGES];
    __shared__ int failed[2][2];  // by team and the parity of its stages: set before a stage's first barrier, read after it
    const int part = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, team = TEAMS == 1 ? 0 : tid / SD_TEAM_THREADS, warp = (tid >> 5) % SD_WARPS, lane = tid & 31, r8 = lane >> 2, q2 = lane & 3;
    if (tid == 0) {
        for (int s = 0; s < p.stages; s++) tc::mbar_init(&full[s], 1), asked[s] = -1;
        failed[0][0] = failed[0][1] = failed[1][0] = failed[1][1] = 0;
        tc::mbar_init_fence();
        tc::tma_prefetch_map(&map_k), tc::tma_prefetch_map(&map_v);
    }
    for (int e = tid; e < H * sm.rows_w; e += SD_TEAM_THREADS * TEAMS) {  // (columns that no head has: zeros, for weights of zero)
        const int h = e / sm.rows_w, g = e - h * sm.rows_w;
        mix_s[h * sm.pitch_m + g] = g >= H ? 0.0f : p.mix ? p.mix[h * H + g] : h == g ? 1.0f : 0.0f;
    }
    for (int e = H * sm.pitch_w + tid; e < sm.w / 4; e += SD_TEAM_THREADS * TEAMS) a_s[e] = a_s[sm.w / 4 + e] = 0.0f;
    if (tid < H) head_s[tid] = sigmoid_head(p.scale, p.softcap, p.slopes ? p.slopes[tid] : 0.0f, p.shift ? p.shift[tid] : 0.0f);
    __syncthreads();
    pdl_wait();
    const int seq = p.token_seq[t];
    if (seq < 0) return;
    const int pos = p.token_pos[t], slot = p.seq_slot[seq], span = sd_span(pos + 1, p.n_parts, kp), first = part * span;
    if (first > pos) return;  // (the fold knows how many parts a row has)
    const int n_keys = min(span, pos + 1 - first), n_st = (n_keys + kp - 1) / kp, box = kp * 128;
    // a stage's boxes, keys and values of every eighth kv head a warp, so that no warp falls behind the others; one thread says
    // how many bytes are to come (some may have come by then). A stage lies within a page (kp divides its PAGE tokens). Stage st lies
    // in place st % stages of the ring; the team that has read it asks for stage st + stages.
    auto issue = [&](int st, int to_stage) {
        const int j = first + st * kp;
        uint64_t *const bar = &full[to_stage];
        if (warp == 0 && lane == 0) {
            tc::mbar_expect_tx(bar, sm.stage);
            __threadfence_block();
            asked[to_stage] = st;
        }
        if (lane == 0) {
            const int page = p.cache.page_table[(long long)slot * p.cache.table_width + j / PAGE];
            uint8_t *const base = ring + to_stage * sm.stage;
            for (int g = warp; g < G; g += SD_WARPS) {
                const int row = (page * G + g) * PAGE + j % PAGE;
                uint8_t *const k = base + g * sm.k_boxes * box, *const v = base + (G * sm.k_boxes + g * sm.v_boxes) * box;
                for (int b = 0; b < sm.k_boxes; b++) tc::tma_load_2d(k + b * box, &map_k, b * 64, row, bar);
                for (int b = 0; b < sm.v_boxes; b++) tc::tma_load_2d(v + b * box, &map_v, b * 64, row, bar);
            }
        }
        __syncwarp();
    };
    for (int st = team; st < n_st && st < p.stages; st += TEAMS) issue(st, st);
    const int d16 = (D + 15) / 16 * 16, tiles_log = kp > 32 ? 2 : kp > 16 ? 1 : 0, half15 = kp > 8 ? 15 : 7;
    const bool capped = p.softcap > 0.0f;
    const __nv_bfloat16 *qg = p.q + (long long)t * p.q_row;
    for (int e = tid; e < H * (d16 / 8); e += SD_TEAM_THREADS * TEAMS) {
        const int h = e / (d16 / 8), d = (e - h * (d16 / 8)) * 8;
        *(uint4 *)(q_s + h * sm.pitch_q + d) = d < D ? *(const uint4 *)(qg + h * D + d) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();

    const int col_tiles = (VD + 15) / 16, units = G * col_tiles, per_warp = (units + SD_WARPS - 1) / SD_WARPS, u0 = warp * per_warp;
    const int g0 = u0 / col_tiles, ct0 = u0 - g0 * col_tiles;
    // a lane's piece of 16 bytes under the swizzle: keys as rows, values transposed
    const uint32_t x_a = ((lane >> 4) ^ (lane & 7)) << 4, x_v = (((lane >> 3) & 1) ^ (lane & 7)) << 4;
    float o[UNITS][NT][4];
#pragma unroll
    for (int i = 0; i < UNITS; i++)
#pragma unroll
        for (int c = 0; c < NT; c++) o[i][c][0] = o[i][c][1] = o[i][c][2] = o[i][c][3] = 0.0f;

    auto meet = [&]() {  // the team's warps
        if (TEAMS == 1) __syncthreads();
        else {
            __syncwarp();  // (the barrier counts whole warps: lanes that waited or took other ways are together again)
            asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "n"(SD_TEAM_THREADS) : "memory");
        }
    };
    float *const weights = a_s + team * (sm.w / 4);
    int s = team, phase = 0, turn = 0;  // the stage's place in the ring, its barrier's phase, the parity of the team's stages
    bool bad = false;
    for (int st = team; st < n_st; st += TEAMS, turn ^= 1) {
        const int j0 = first + st * kp, nv = min(kp, n_keys - st * kp);
        const uint32_t k_s = tc::smem_addr(ring + s * sm.stage), v_s = k_s + G * sm.k_boxes * box;
        __syncwarp();
        if (!(sd_asked(&asked[s], st) && tc::mbar_wait(&full[s], phase))) failed[team][turn] = 1;
        // scores: a warp takes a kv head and 16 keys at a time
        // (a stage of 8 keys fills half of a tile: the other half repeats them and is dropped, here and below)
        for (int u = warp; u < G << tiles_log; u += SD_WARPS) {
            const int g = u >> tiles_log, key = (u - (g << tiles_log)) * 16;
            float c[NT][4];
#pragma unroll
            for (int i = 0; i < NT; i++) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.0f;
            uint32_t kb = k_s + g * sm.k_boxes * box + (key + (lane & half15)) * 128;
            const uint32_t *qr[NT];  // (columns beyond the group's heads repeat a head and are dropped)
#pragma unroll
            for (int i = 0; i < NT; i++) qr[i] = (const uint32_t *)(q_s + (g * R + min(8 * i + r8, R - 1)) * sm.pitch_q) + q2;
            for (int left = d16 / 16; left > 0; left -= 4, kb += box) {
#pragma unroll
                for (int c4 = 0; c4 < 4; c4++) {
                    if (c4 < left) {
                        uint32_t a[4];
                        ldsm_x4(kb + (x_a ^ (c4 << 5)), a[0], a[1], a[2], a[3]);
#pragma unroll
                        for (int i = 0; i < NT; i++) mma_bf16(c[i], a, qr[i][8 * c4], qr[i][8 * c4 + 4]);
                    }
                }
#pragma unroll
                for (int i = 0; i < NT; i++) qr[i] += 32;
            }
            // the weights of this lane's keys (rows) and heads (columns)
            const float back = (float)(pos - j0 - key - r8);
            const bool in_a = key + r8 < nv, in_b = key + r8 + 8 < nv;
#pragma unroll
            for (int i = 0; i < NT; i++) {
                const int hl = 8 * i + 2 * q2;
                if (hl >= R) continue;
                const SigmoidHead e = head_s[g * R + hl], f = head_s[g * R + (hl + 1 < R ? hl + 1 : hl)];
                c[i][0] = in_a ? sigmoid_of(capped, e, c[i][0], fmaf(e.slope, back, e.base)) : 0.0f;
                c[i][1] = in_a ? sigmoid_of(capped, f, c[i][1], fmaf(f.slope, back, f.base)) : 0.0f;
                c[i][2] = in_b ? sigmoid_of(capped, e, c[i][2], fmaf(e.slope, back - 8.0f, e.base)) : 0.0f;
                c[i][3] = in_b ? sigmoid_of(capped, f, c[i][3], fmaf(f.slope, back - 8.0f, f.base)) : 0.0f;
                float *to = weights + (g * R + hl) * sm.pitch_w + key + r8;
                if (hl < R) to[0] = c[i][0];
                if (hl + 1 < R) to[sm.pitch_w] = c[i][1];
                if (kp > 8) {
                    if (hl < R) to[8] = c[i][2];
                    if (hl + 1 < R) to[sm.pitch_w + 8] = c[i][3];
                }
            }
        }
        if (nv < kp) {  // the last stage: rows beyond the token's key hold what the page held; they count as zeros
            const int per = sm.v_boxes * 8;
            for (int e = tid - team * SD_TEAM_THREADS; e < G * (kp - nv) * per; e += SD_TEAM_THREADS) {
                const int row = e / per, c = e - row * per, g = row / (kp - nv), key = nv + row - g * (kp - nv);
                *(uint4 *)(ring + s * sm.stage + (G * sm.k_boxes + g * sm.v_boxes + (c >> 3)) * box + key * 128 + (c & 7) * 16) = make_uint4(0, 0, 0, 0);
            }
        }
        meet();  // the stage's weights are there
        if (failed[team][turn]) {  // a copy did not come: let the team's copies still in flight land (or run out of time)
            for (int i = 0; i < p.stages; i++)
                if (asked[i] >= 0) tc::mbar_wait(&full[i], (asked[i] / p.stages) & 1);
            bad = true;
            break;
        }
        // values: this warp's tiles, which follow one another, so that a kv head's weights are split once
        for (int key = 0; key < kp && key < nv; key += 16) {
            int g = g0, ct = ct0, have = -1;
            const uint32_t one = ONE ? g0 * sm.v_boxes * box : 0;
            const uint32_t vb = v_s + (key + (((lane & 7) + (lane >> 4) * 8) & half15)) * 128;
            uint32_t b0[NT][3], b1[NT][3];
#pragma unroll
            for (int i = 0; i < UNITS; i++) {
                if (!ONE && (u0 + i >= units || i >= per_warp)) break;
                if (ONE ? i == 0 : g != have) {
                    have = g;
#pragma unroll
                    for (int c = 0; c < NT; c++) {
                        const int hl = 8 * c + r8;
                        const float *w = weights + key + 2 * q2, *m = mix_s + (g * R + (hl < R ? hl : 0)) * sm.pitch_m;
                        float2 lo = make_float2(0.0f, 0.0f), hi = lo;
                        if (hl < R) {
                            for (int from = 0; from < sm.rows_w; from += 4, w += 4 * sm.pitch_w) {
                                const float4 mx = *(const float4 *)(m + from);
                                const float by[4] = {mx.x, mx.y, mx.z, mx.w};
#pragma unroll
                                for (int u = 0; u < 4; u++) {
                                    const float2 x = *(const float2 *)(w + u * sm.pitch_w);
                                    lo.x = fmaf(by[u], x.x, lo.x), lo.y = fmaf(by[u], x.y, lo.y);
                                    if (kp > 8) {
                                        const float2 y = *(const float2 *)(w + u * sm.pitch_w + 8);
                                        hi.x = fmaf(by[u], y.x, hi.x), hi.y = fmaf(by[u], y.y, hi.y);
                                    }
                                }
                            }
                        }
                        split3_pair(lo.x, lo.y, b0[c]), split3_pair(hi.x, hi.y, b1[c]);
                    }
                }
                // rows: 16 value columns; the fragment is the transposed tile of 16 keys x 16 columns
                uint32_t a[4];
                if (ONE) ct = i;
                ldsm_x4_t(vb + (ONE ? one + (i >> 2) * box : (g * sm.v_boxes + (ct >> 2)) * box) + (x_v ^ ((ct & 3) << 5)), a[0], a[1], a[2], a[3]);
#pragma unroll
                for (int c = 0; c < NT; c++)
#pragma unroll
                    for (int k = 0; k < 3; k++) mma_bf16(o[i][c], a, b0[c][k], b1[c][k]);
                if (!ONE && ++ct == col_tiles) ct = 0, g++;
            }
        }
        meet();  // the stage and the weights are done with
        if (st + p.stages < n_st) issue(st + p.stages, s);
        s += TEAMS;
        if (s >= p.stages) s -= p.stages, phase ^= 1;
    }
    if (bad && lane == 0 && warp == 0) atomicOr(p.status + 2, 1);
    if (TEAMS == 2) {  // the second team's sums, a warp's beside those of the first team's warp that has the same tiles
        float4 *const sums = (float4 *)ring + warp * (UNITS * NT * 32) + lane;
        __syncthreads();  // (the ring is done with)
        if (team == 1) {
#pragma unroll
            for (int i = 0; i < UNITS; i++)
#pragma unroll
                for (int c = 0; c < NT; c++) sums[(i * NT + c) * 32] = make_float4(o[i][c][0], o[i][c][1], o[i][c][2], o[i][c][3]);
        }
        __syncthreads();
        if (team == 1) return;
#pragma unroll
        for (int i = 0; i < UNITS; i++) {
#pragma unroll
            for (int c = 0; c < NT; c++) {
                const float4 v = sums[(i * NT + c) * 32];
                o[i][c][0] += v.x, o[i][c][1] += v.y, o[i][c][2] += v.z, o[i][c][3] += v.w;
            }
        }
    }
    float *dst = p.parts + ((long long)t * p.n_parts + part) * H * VD;
    int g = g0, ct = ct0;
#pragma unroll
    for (int i = 0; i < UNITS; i++) {
        if (u0 + i >= units || i >= per_warp) break;
#pragma unroll
        for (int c = 0; c < NT; c++) {
            const int hl = 8 * c + 2 * q2, col = ct * 16 + r8;
            float *to = dst + (long long)(g * R + hl) * VD + col;
            if (hl < R) {
                if (col < VD) to[0] = o[i][c][0];
                if (col + 8 < VD) to[8] = o[i][c][2];
            }
            if (hl + 1 < R) {
                if (col < VD) to[VD] = o[i][c][1];
                if (col + 8 < VD) to[VD + 8] = o[i][c][3];
            }
        }
        if (++ct == col_tiles) ct = 0, g++;
    }
}

// out[t] = the sum of a row's parts: four columns a thread, 8 runs of parts side by side, added in order.
__global__ void __launch_bounds__(256) attention_sigmoid_fold_kernel(SigmoidDecode p) {
    __shared__ float4 sums[8][32];
    const int t = blockIdx.y, lane = threadIdx.x & 31, run = threadIdx.x >> 5, width = p.n_heads * p.v_dim;
    const int c = (blockIdx.x * 32 + lane) * 4;
    pdl_wait();
    const int seq = p.token_seq[t];
    float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (seq >= 0 && c < width) {
        const int keys = p.token_pos[t] + 1, span = sd_span(keys, p.n_parts, p.kp), n = (keys + span - 1) / span;
        const float *src = p.parts + (long long)t * p.n_parts * width + c;
        for (int i = run; i < n; i += 32) {  // (four of this run's parts on their way together)
            float4 v[4];
#pragma unroll
            for (int k = 0; k < 4; k++)
                v[k] = i + 8 * k < n ? *(const float4 *)(src + (long long)(i + 8 * k) * width) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int k = 0; k < 4; k++) sum.x += v[k].x, sum.y += v[k].y, sum.z += v[k].z, sum.w += v[k].w;
        }
    }
    sums[run][lane] = sum;
    __syncthreads();
    if (run > 0 || c >= width) return;
    for (int i = 1; i < 8; i++) {
        const float4 v = sums[i][lane];
        sum.x += v.x, sum.y += v.y, sum.z += v.z, sum.w += v.w;
    }
    const __nv_bfloat162 lo = __floats2bfloat162_rn(sum.x, sum.y), hi = __floats2bfloat162_rn(sum.z, sum.w);
    *(uint2 *)(p.out + (long long)t * width + c) = make_uint2(*(const uint32_t *)&lo, *(const uint32_t *)&hi);
}

// Stages of a ring for these sizes: the most keys a stage holds (8, 16, 32 or 64; a stage of at most about 64 KB unless 8 keys
// are more) and how many stages fit; 0 if not one does.
static int sd_plan(int H, int G, int D, int VD, int &kp, int &stages) {
    kp = 64;
    while (kp > 8 && SigmoidDecodeSmem(H, G, D, VD, kp, 1).stage > 66 * 1024) kp /= 2;
    for (stages = SD_MAX_STAGES; stages >= 1; stages--)
        if (SigmoidDecodeSmem(H, G, D, VD, kp, stages).total <= 225 * 1024) return 1;
    return 0;
}

// The parts a row of a step of n_tokens rows is cut into, so that the step is about a CTA an SM (what the caller's scratch memory is sized by); 0: these sizes
// are not taken.
extern "C" int abk_attention_sigmoid_decode_parts(int n_tokens, int n_heads, int n_kv_heads, int head_dim, int v_dim, int max_keys) {
    if (n_heads < 1 || n_kv_heads < 1 || n_heads % n_kv_heads || head_dim % 8 || v_dim % 8 || head_dim < 8 || v_dim < 8) return 0;
    if (n_tokens < 1 || n_tokens > 65535 || n_heads > 256 || n_heads / n_kv_heads > 16 || max_keys < 1) return 0;
    const int nt = n_heads / n_kv_heads > 8 ? 2 : 1, units = (n_kv_heads * ((v_dim + 15) / 16) + SD_WARPS - 1) / SD_WARPS;
    if (units * nt > 32) return 0;
    int kp, stages;
    if (!sd_plan(n_heads, n_kv_heads, head_dim, v_dim, kp, stages)) return 0;
    int parts = abk_sm_count() / n_tokens, most = (max_keys + 2 * kp - 1) / (2 * kp);
    if (parts > most) parts = most;
    return parts < 1 ? 1 : parts;
}

// n_parts: what abk_attention_sigmoid_decode_parts said; parts: float32 scratch of n_tokens * n_parts * n_heads * v_dim.
// pool_rows: rows of head_dim (v_dim) elements the key (value) pool has. status word 2 is set if a wait ran out.
extern "C" int abk_attention_sigmoid_decode(const void *q, long long q_row, void *out, int n_tokens, int n_heads, int n_kv_heads,
                                            int head_dim, int v_dim, float scale, float softcap, const float *slopes,
                                            const float *shift, const float *mix, const int *token_seq, const int *token_pos,
                                            const int *seq_slot, const void *k_pool, const void *v_pool, long long pool_rows,
                                            const int *page_table, int table_width, int tokens_per_page, int n_parts,
                                            float *parts, int *status, void *stream) {
    if (n_tokens <= 0) return 0;
    if (!abk_attention_sigmoid_decode_parts(n_tokens, n_heads, n_kv_heads, head_dim, v_dim, 1) || n_parts < 1 || n_parts > 65535)
        ABK_REFUSE("attention_sigmoid_decode: %d heads of %d over %d kv heads with values of %d", n_heads, head_dim, n_kv_heads, v_dim);
    if (tokens_per_page != PAGE || pool_rows > 0x7fffffffLL) ABK_REFUSE("attention_sigmoid_decode: pages of %d tokens", tokens_per_page);
    if ((((uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)parts | (uintptr_t)q) & 15) || q_row % 8 || (uintptr_t)out & 7)
        ABK_REFUSE("attention_sigmoid_decode: the cache's pools and the output must be 16-byte aligned");
    SigmoidDecode p;
    p.q = (const __nv_bfloat16 *)q, p.q_row = q_row, p.parts = parts, p.out = (__nv_bfloat16 *)out;
    p.n_heads = n_heads, p.n_kv_heads = n_kv_heads, p.head_dim = head_dim, p.v_dim = v_dim, p.scale = scale, p.softcap = softcap;
    p.slopes = slopes, p.shift = shift, p.mix = mix, p.token_seq = token_seq, p.token_pos = token_pos, p.seq_slot = seq_slot;
    p.cache.page_table = page_table, p.cache.table_width = table_width, p.cache.ring_pages = 0;
    p.cache.tokens_per_page = tokens_per_page, p.cache.pinned_pages = 0;
    p.n_parts = n_parts, p.status = status;
    sd_plan(n_heads, n_kv_heads, head_dim, v_dim, p.kp, p.stages);
    CUtensorMap mk, mv;
    int rc = tmap::bf16_rows_of_128_bytes(k_pool, pool_rows, head_dim, head_dim, p.kp, &mk);
    if (!rc) rc = tmap::bf16_rows_of_128_bytes(v_pool, pool_rows, v_dim, v_dim, p.kp, &mv);
    if (rc) return rc;
    const int smem = SigmoidDecodeSmem(n_heads, n_kv_heads, head_dim, v_dim, p.kp, p.stages).total;
    const int units = (n_kv_heads * ((v_dim + 15) / 16) + SD_WARPS - 1) / SD_WARPS, nt = n_heads / n_kv_heads > 8 ? 2 : 1;
    const dim3 grid(n_parts, n_tokens);
    cudaStream_t s = (cudaStream_t)stream;
#define SD_LAUNCH(UNITS, NT, ONE, TEAMS)                                                                                             \
    do {                                                                                                                             \
        cudaError_t e = abk_allow_shared_memory((const void *)attention_sigmoid_decode_kernel<UNITS, NT, ONE, TEAMS>, smem);         \
        if (e != cudaSuccess) return (int)e;                                                                                         \
        abk_launch(attention_sigmoid_decode_kernel<UNITS, NT, ONE, TEAMS>, grid, dim3(SD_TEAM_THREADS * TEAMS), (size_t)smem, s, mk, mv, p); \
    } while (0)
    const bool two = p.stages >= 2;  // (a ring of one stage is read by one team)
    if (nt == 2) SD_LAUNCH(16, 2, false, 1);
    else if (two && n_kv_heads == 8 && v_dim > 112 && v_dim <= 128) SD_LAUNCH(8, 1, true, 2);
    else if (two && units <= 8) SD_LAUNCH(8, 1, false, 2);
    else if (two && units <= 16) SD_LAUNCH(16, 1, false, 2);
    else SD_LAUNCH(32, 1, false, 1);
#undef SD_LAUNCH
    rc = ABK_LAUNCH_RESULT();
    if (rc) return rc;
    abk_launch(attention_sigmoid_fold_kernel, dim3((n_heads * v_dim / 4 + 31) / 32, n_tokens), dim3(256), 0, s, p);
    return ABK_LAUNCH_RESULT();
}
