// Router epilogue: scores, bias-corrected choice, top-k, renormalisation and scaling, all float32.
//
// sigmoid form (python/freetoken/models/minimax_m3/moe.py:71-81): s = sigmoid(logits); the experts
// are chosen by s + bias, weighted by the unbiased s, divided by their sum (+1e-20) and multiplied by
// the scaling factor.  softmax form (python/freetoken/moe/fused.py:27-31): s = softmax(logits).
// Raw forms leave the chosen scores as they are.  Experts may form equal groups of neighbours of which only the best few
// (by their largest choice) may be chosen from.
// One warp per token; the largest choice goes first and the lower expert index wins a tie.
// For long steps the logits are a library matrix product in float32, as in the reference (F.linear),
// and router_topk_kernel takes them; for short steps moe_route_kernel computes them itself and also
// sorts the routes by expert, all in one launch.
#include "common.cuh"

namespace ftk {

constexpr int kRouterWarps = 4;

// A token's logit of expert e: the row holds n_parts blocks of n_experts values that are added in their
// order (one block: the logits themselves; three: the products of the activations with the three
// bfloat16 pieces of the float32 router weights, largest first).
__device__ __forceinline__ float logit_of(const float* __restrict__ row, int e, int part_stride, int n_parts) {
  float v = __ldcg(row + e);
  for (int q = 1; q < n_parts; ++q) v += __ldcg(row + (size_t)q * part_stride + e);
  return v;
}

// What a token's routing leaves beside ids and weights (one warp): the sum of the chosen experts' weights that belong
// to ids from n_real on (experts without tensors), and the sigmoid of the logit behind the experts' (1 without one).
__device__ __forceinline__ void token_aux(const float* __restrict__ row, int part_stride, int n_parts, int n_experts, int n_extra,
                                          int n_real, const int32_t* ids, const float* weights, int top_k, float* __restrict__ aux) {
  const int lane = threadIdx.x & 31;
  __syncwarp();  // the warp's own stores of ids and weights
  float sum = 0.f;
  for (int j = lane; j < top_k; j += 32) sum += ids[j] >= n_real ? weights[j] : 0.f;
  sum = warp_sum(sum);
  if (lane == 0) {
    aux[0] = sum;
    aux[1] = n_extra ? 1.f / (1.f + expf(-logit_of(row, n_experts, part_stride, n_parts))) : 1.f;
  }
}

// Experts in `count` equal groups of neighbours, of which the `keep` with the largest choice in them are open (count 1: all).
struct RouteGroups {
  int count, keep;
};

// What the chosen scores are divided by: nothing (1) in the raw forms.
__device__ __forceinline__ float weight_denominator(int scoring, float wsum) {
  if (scoring == FTK_SCORE_SIGMOID_RAW || scoring == FTK_SCORE_SOFTMAX_RAW) return 1.f;
  return scoring == FTK_SCORE_SOFTMAX_OF_CHOSEN ? wsum : wsum + 1e-20f;
}

// The largest of c[0 .. n_experts) whose group is not in `closed` (a bit per group; size 0: no groups), by one warp; the
// lowest index of equal ones; 0x7fffffff when every value is NaN or -inf.
__device__ __forceinline__ int best_choice(const float* c, int n_experts, int size, unsigned long long closed) {
  float best = -INFINITY;
  int bi = 0x7fffffff;
  for (int e = threadIdx.x & 31; e < n_experts; e += 32) {
    const float v = size && (closed >> (e / size) & 1) ? -INFINITY : c[e];
    if (v > best) {  // ascending e within a lane: the first of equal values stays
      best = v;
      bi = e;
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ob = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ob > best || (ob == best && oi < bi)) {
      best = ob;
      bi = oi;
    }
  }
  return bi;
}

// Scores, choice and weights of one token, by one warp.  `s` and `c` hold n_experts floats each.
__device__ __forceinline__ void route_token(const float* __restrict__ row, int part_stride, int n_parts, const float* __restrict__ bias,
                                            int n_experts, RouteGroups groups, int top_k, int scoring, float scale, float* s, float* c,
                                            int32_t* __restrict__ ids, float* __restrict__ weights,
                                            int32_t* ids_copy) {
  const int lane = threadIdx.x & 31;
  // softmax over the chosen experts of logit + bias: the bias joins the logit, the softmax over all experts keeps
  // the order, and dividing by the chosen experts' sum below leaves the softmax over them alone
  const float* pre = scoring == FTK_SCORE_SOFTMAX_OF_CHOSEN ? bias : nullptr;
  if (pre) bias = nullptr;
  if (scoring == FTK_SCORE_SIGMOID || scoring == FTK_SCORE_SIGMOID_RAW) {
    for (int e = lane; e < n_experts; e += 32) s[e] = 1.f / (1.f + expf(-logit_of(row, e, part_stride, n_parts)));
  } else {
    float mx = -INFINITY;
    for (int e = lane; e < n_experts; e += 32) mx = fmaxf(mx, logit_of(row, e, part_stride, n_parts) + (pre ? pre[e] : 0.f));
    mx = warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < n_experts; e += 32) {
      const float v = expf(logit_of(row, e, part_stride, n_parts) + (pre ? pre[e] : 0.f) - mx);
      s[e] = v;
      sum += v;
    }
    sum = warp_sum(sum);
    for (int e = lane; e < n_experts; e += 32) s[e] = s[e] / sum;
  }
  for (int e = lane; e < n_experts; e += 32) c[e] = bias ? s[e] + bias[e] : s[e];
  __syncwarp();
  if (groups.keep < groups.count) {  // the best expert of all is in the best group, the best of the rest in the next, ...
    const int size = n_experts / groups.count;
    unsigned long long open = 0;
    for (int g = 0; g < groups.keep; ++g) {
      const int e = best_choice(c, n_experts, size, open);
      if (e != 0x7fffffff) open |= 1ull << (e / size);
    }
    __syncwarp();
    for (int e = lane; e < n_experts; e += 32)
      if (!(open >> (e / size) & 1)) c[e] = -INFINITY;
    __syncwarp();
  }
  float wsum = 0.f;
  for (int j = 0; j < top_k; ++j) {
    int bi = best_choice(c, n_experts, 0, 0);
    if (bi == 0x7fffffff) bi = 0;  // every remaining choice is NaN or -inf
    const float w = s[bi];
    wsum += w;
    if (lane == 0) {
      ids[j] = bi;
      if (ids_copy) ids_copy[j] = bi;
      weights[j] = w;
      c[bi] = -INFINITY;
    }
    __syncwarp();
  }
  const float denom = weight_denominator(scoring, wsum);
  for (int j = lane; j < top_k; j += 32) weights[j] = weights[j] / denom * scale;
}

// The same with the token's scores in registers (n_experts <= 32 * PER): the largest remaining choice
// is found with two warp reductions, first over the values (as order-preserving integers, NaN lowest),
// then over the indices of those that have it.  Same results as route_token.
__device__ __forceinline__ unsigned int order_key(float v) {
  if (v != v) return 0u;
  const unsigned int u = __float_as_uint(v + 0.f);  // -0 becomes +0
  return (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}

template <int PER>
__device__ __forceinline__ void route_token_regs(const float* __restrict__ row, int part_stride, int n_parts, const float* __restrict__ bias,
                                                 int n_experts, RouteGroups groups, int top_k, int scoring, float scale, float* wbuf,
                                                 int32_t* __restrict__ ids, float* __restrict__ weights,
                                                 int32_t* ids_copy) {
  const int lane = threadIdx.x & 31;
  float sv[PER];
  unsigned int key[PER];
#pragma unroll
  for (int q = 0; q < PER; ++q) {
    const int e = q * 32 + lane;
    sv[q] = e < n_experts ? logit_of(row, e, part_stride, n_parts) : -INFINITY;
  }
  if (scoring == FTK_SCORE_SOFTMAX_OF_CHOSEN) {  // the bias joins the logit (see route_token)
    if (bias) {
#pragma unroll
      for (int q = 0; q < PER; ++q) {
        const int e = q * 32 + lane;
        if (e < n_experts) sv[q] += bias[e];
      }
    }
    bias = nullptr;
  }
  if (scoring == FTK_SCORE_SIGMOID || scoring == FTK_SCORE_SIGMOID_RAW) {
#pragma unroll
    for (int q = 0; q < PER; ++q) sv[q] = 1.f / (1.f + expf(-sv[q]));
  } else {
    float mx = -INFINITY;
#pragma unroll
    for (int q = 0; q < PER; ++q) mx = fmaxf(mx, sv[q]);
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      sv[q] = q * 32 + lane < n_experts ? expf(sv[q] - mx) : 0.f;
      sum += sv[q];
    }
    // the sum runs over experts in the order route_token takes them: lane by lane, then across lanes
    sum = warp_sum(sum);
#pragma unroll
    for (int q = 0; q < PER; ++q) sv[q] = sv[q] / sum;
  }
  const unsigned int floor_key = order_key(-INFINITY);  // never chosen: -inf and NaN
#pragma unroll
  for (int q = 0; q < PER; ++q) {
    const int e = q * 32 + lane;
    key[q] = e < n_experts ? order_key(bias ? sv[q] + bias[e] : sv[q]) : 0u;
  }
  if (groups.keep < groups.count) {  // (see route_token)
    const int size = n_experts / groups.count;
    unsigned int open = 0;  // a bit per slot of the lane
    for (int g = 0; g < groups.keep; ++g) {
      unsigned int best = 0u;
      int slot = 0;
#pragma unroll
      for (int q = 0; q < PER; ++q)
        if (key[q] > best && !(open >> q & 1)) {
          best = key[q];
          slot = q;
        }
      const unsigned int top = __reduce_max_sync(0xffffffffu, best);
      if (top <= floor_key) break;
      const int first = (int)__reduce_min_sync(0xffffffffu, best == top ? (unsigned)(slot * 32 + lane) : 0x7fffffffu) / size * size;
#pragma unroll
      for (int q = 0; q < PER; ++q) {
        const int e = q * 32 + lane;
        if (e >= first && e < first + size) open |= 1u << q;
      }
    }
#pragma unroll
    for (int q = 0; q < PER; ++q)
      if (!(open >> q & 1)) key[q] = 0u;
  }
  float wsum = 0.f;
  for (int j = 0; j < top_k; ++j) {
    unsigned int best = 0u;
    int slot = 0;
#pragma unroll
    for (int q = 0; q < PER; ++q)
      if (key[q] > best) {
        best = key[q];
        slot = q;
      }
    const unsigned int top = __reduce_max_sync(0xffffffffu, best);
    int bi = 0;
    if (top > floor_key) bi = (int)__reduce_min_sync(0xffffffffu, best == top ? (unsigned)(slot * 32 + lane) : 0x7fffffffu);
    const int owner = bi & 31, oslot = bi >> 5;
    float mine = 0.f;
#pragma unroll
    for (int q = 0; q < PER; ++q)
      if (q == oslot) mine = sv[q];
    const float w = __shfl_sync(0xffffffffu, mine, owner);
    wsum += w;
    if (lane == owner && top > floor_key) {
#pragma unroll
      for (int q = 0; q < PER; ++q)
        if (q == oslot) key[q] = 0u;
    }
    if (lane == 0) {
      ids[j] = bi;
      if (ids_copy) ids_copy[j] = bi;
      wbuf[j] = w;
    }
  }
  __syncwarp();
  const float denom = weight_denominator(scoring, wsum);
  for (int j = lane; j < top_k; j += 32) weights[j] = wbuf[j] / denom * scale;
  __syncwarp();
}

// One token by one warp, in registers where the experts fit; `s` holds 2 * n_experts floats.
__device__ __forceinline__ void route_one(const float* __restrict__ row, int part_stride, int n_parts, const float* __restrict__ bias, int n_experts,
                                          RouteGroups groups, int top_k, int scoring, float scale, float* s, int32_t* __restrict__ ids,
                                          float* __restrict__ weights, int32_t* ids_copy) {
  if (n_experts <= 128)
    route_token_regs<4>(row, part_stride, n_parts, bias, n_experts, groups, top_k, scoring, scale, s, ids, weights, ids_copy);
  else if (n_experts <= 256)
    route_token_regs<8>(row, part_stride, n_parts, bias, n_experts, groups, top_k, scoring, scale, s, ids, weights, ids_copy);
  else if (n_experts <= 512)
    route_token_regs<16>(row, part_stride, n_parts, bias, n_experts, groups, top_k, scoring, scale, s, ids, weights, ids_copy);
  else
    route_token(row, part_stride, n_parts, bias, n_experts, groups, top_k, scoring, scale, s, s + n_experts, ids, weights, ids_copy);
}

__global__ void router_topk_kernel(const float* __restrict__ logits, int n_parts, const float* __restrict__ bias,
                                   int n_tokens, int n_experts, int top_k, int scoring, float scale,
                                   int32_t* __restrict__ ids, float* __restrict__ weights, int n_extra, int n_pad, int n_real,
                                   float* __restrict__ aux, RouteGroups groups) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5;
  const int t = blockIdx.x * kRouterWarps + warp;
  if (t >= n_tokens) return;
  float* s = sm + (size_t)warp * 2 * n_experts;  // unbiased scores
  const int stride = n_experts + n_extra + n_pad;
  const float* row = logits + (size_t)t * n_parts * stride;
  route_one(row, stride, n_parts, bias, n_experts, groups, top_k, scoring, scale, s, ids + (size_t)t * top_k,
            weights + (size_t)t * top_k, nullptr);
  if (aux)
    token_aux(row, stride, n_parts, n_experts, n_extra, n_real, ids + (size_t)t * top_k, weights + (size_t)t * top_k, top_k,
              aux + (size_t)t * 2);
}

// The whole routing of a small step in one launch: router logits (a float32 matrix-vector product
// per token, python/freetoken/models/minimax_m3/moe.py:71-73), then, in the block that finishes
// last, the choice of every token (route_one) and the sort of the routes by expert (what moe_permute
// does).  A block holds kRouteExperts experts; its warps share their weight rows (a thread's piece of
// them is on its way before the kernel waits for the one before it) and add their parts in a fixed
// order, so a token's logits never depend on the batch.  Blocks count their arrival in
// g_route_arrivals; nobody waits for anybody.
constexpr int kRouteWarps = 24;   // all of them share the block's weight rows, each a part of the width
constexpr int kRouteExperts = 2;  // experts per block: a token's activations are loaded once for all of them
constexpr int kRouteTokens = 8;   // tokens per pass over the weight rows
constexpr int kRouteVals = kRouteExperts * kRouteTokens;  // sums a thread carries
static_assert(kRouteVals == 16, "warp_sum16 adds sixteen values per lane");
__device__ unsigned int g_route_arrivals = 0;

// Sixteen sums over the warp with sixteen shuffles: the lanes swap halves of what they carry and keep
// the other half, four times; lanes 2 i and 2 i + 1 end up with the warp's sum of value i.
__device__ __forceinline__ float warp_sum16(float (&v)[16], int lane) {
  const bool b4 = lane & 16, b3 = lane & 8, b2 = lane & 4, b1 = lane & 2;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const float give = b4 ? v[i] : v[i + 8], keep = b4 ? v[i + 8] : v[i];
    v[i] = keep + __shfl_xor_sync(0xffffffffu, give, 16);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float give = b3 ? v[i] : v[i + 4], keep = b3 ? v[i + 4] : v[i];
    v[i] = keep + __shfl_xor_sync(0xffffffffu, give, 8);
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const float give = b2 ? v[i] : v[i + 2], keep = b2 ? v[i + 2] : v[i];
    v[i] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
  }
  {
    const float give = b1 ? v[0] : v[1], keep = b1 ? v[1] : v[0];
    v[0] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
}

__global__ void __launch_bounds__(kRouteWarps * 32)
moe_route_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ bias,
                 int n_tokens, int hidden, int n_experts, int top_k, int scoring, float scale,
                 float* __restrict__ logits, int32_t* __restrict__ ids, float* __restrict__ weights,
                 int32_t* __restrict__ counts, int32_t* __restrict__ offsets, int32_t* __restrict__ routes,
                 int32_t* __restrict__ pos, int do_sort, int n_extra, int n_real, float* __restrict__ aux, RouteGroups groups) {
  const int n_rows = n_experts + n_extra;  // rows of the weight, logits of a token
  extern __shared__ float sm[];
  __shared__ float part[kRouteVals][kRouteWarps + 1];
  __shared__ bool last;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int e0 = blockIdx.x * kRouteExperts;
  const int h4 = hidden >> 2;
  const float4* w4 = reinterpret_cast<const float4*>(w);
  const float4* x4 = reinterpret_cast<const float4*>(x);
  // the router's weights never depend on the kernel before: a thread's first pieces of them are on
  // their way before the wait
  float4 w_first[kRouteExperts];
#pragma unroll
  for (int j = 0; j < kRouteExperts; ++j)
    w_first[j] = tid < h4 ? __ldg(w4 + (size_t)min(e0 + j, n_rows - 1) * h4 + tid) : make_float4(0.f, 0.f, 0.f, 0.f);
  pdl_wait();
  // every block fetches the bias now, under the matrix product, so that the one that turns out to
  // be last does not wait for it
  float* sbias = sm + (size_t)kRouteWarps * 2 * n_experts;
  if (bias)
    for (int i = tid; i < n_experts; i += blockDim.x) sbias[i] = __ldg(bias + i);
  for (int t0 = 0; t0 < n_tokens; t0 += kRouteTokens) {
    const int nt = min(kRouteTokens, n_tokens - t0);
    float acc[kRouteVals];  // [expert][token]
#pragma unroll
    for (int i = 0; i < kRouteVals; ++i) acc[i] = 0.f;
#pragma unroll 2
    for (int i = tid; i < h4; i += kRouteWarps * 32) {
      float4 wv[kRouteExperts], xv[kRouteTokens];
#pragma unroll
      for (int j = 0; j < kRouteExperts; ++j)
        wv[j] = i == tid ? w_first[j] : __ldg(w4 + (size_t)min(e0 + j, n_rows - 1) * h4 + i);
#pragma unroll
      for (int u = 0; u < kRouteTokens; ++u)  // (rows past the step's tokens are never stored: no load for them)
        xv[u] = u < nt ? __ldg(x4 + (size_t)(t0 + u) * h4 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < kRouteExperts; ++j)
#pragma unroll
        for (int u = 0; u < kRouteTokens; ++u) {
          float a = acc[j * kRouteTokens + u];
          a = fmaf(wv[j].x, xv[u].x, a);
          a = fmaf(wv[j].y, xv[u].y, a);
          a = fmaf(wv[j].z, xv[u].z, a);
          a = fmaf(wv[j].w, xv[u].w, a);
          acc[j * kRouteTokens + u] = a;
        }
    }
    const float total = warp_sum16(acc, lane);
    if (!(lane & 1)) part[lane >> 1][warp] = total;
    __syncthreads();
    if (tid < kRouteVals) {
      const int j = tid / kRouteTokens, u = tid % kRouteTokens;
      if (u < nt && e0 + j < n_rows) {
        float v = part[tid][0];
#pragma unroll
        for (int q = 1; q < kRouteWarps; ++q) v += part[tid][q];
        logits[(size_t)(t0 + u) * n_rows + e0 + j] = v;
      }
    }
    __syncthreads();
  }
  if (tid < kRouteVals) __threadfence();
  __syncthreads();
  if (tid == 0) last = atomicAdd(&g_route_arrivals, 1u) == gridDim.x - 1;
  __syncthreads();
  if (!last) return;
  __threadfence();
  // ---- the last block: every token's choice
  const int n_routes = n_tokens * top_k;
  int* sid = reinterpret_cast<int*>(sbias + n_experts);  // n_routes: the routes' experts
  float* s = sm + (size_t)warp * 2 * n_experts;
  for (int t = warp; t < n_tokens; t += kRouteWarps) {
    const float* row = logits + (size_t)t * n_rows;
    route_one(row, n_rows, 1, bias ? sbias : nullptr, n_experts, groups, top_k, scoring, scale, s, ids + (size_t)t * top_k,
              weights + (size_t)t * top_k, do_sort ? sid + (size_t)t * top_k : nullptr);
    if (aux)
      token_aux(row, n_rows, 1, n_experts, n_extra, n_real, ids + (size_t)t * top_k, weights + (size_t)t * top_k, top_k,
                aux + (size_t)t * 2);
  }
  if (!do_sort) {  // the caller's kernels take the routes in token order
    if (tid == 0) g_route_arrivals = 0;
    return;
  }
  __syncthreads();
  // ---- the routes sorted by expert; rows of one expert keep the order of the routes.  A route's
  // place is the number of routes that come before it, an expert's offset the number of routes to
  // experts below it: every thread counts for itself, nothing is scanned or scattered.
  for (int r = tid; r < n_routes; r += blockDim.x) {
    const int e = sid[r];
    int before = 0;
    for (int q = 0; q < n_routes; ++q) {
      const int eq = sid[q];
      before += (eq < e || (eq == e && q < r)) ? 1 : 0;
    }
    routes[before] = r;
    pos[r] = e < n_real ? before : -1;  // (an expert without tensors has no rows)
  }
  for (int i = tid; i <= n_real; i += blockDim.x) {
    int below = 0, same = 0;
    for (int q = 0; q < n_routes; ++q) {
      const int eq = sid[q];
      below += eq < i ? 1 : 0;
      same += eq == i ? 1 : 0;
    }
    offsets[i] = below;
    if (i < n_real) counts[i] = same;
  }
  if (tid == 0) g_route_arrivals = 0;  // every block has arrived: ready for the next launch
}

}  // namespace ftk

using namespace ftk;

// (more than 512 experts are chosen from with a bit per group: at most 64 of them)
static bool groups_ok(int n_experts, int count, int keep, int top_k) {
  return count >= 1 && keep >= 1 && keep <= count && n_experts % count == 0 && (n_experts <= 512 || count <= 64) &&
         (keep == count || top_k <= n_experts / count * keep);
}

extern "C" int ftk_router_topk(const float* logits, int n_parts, const float* bias, int n_tokens, int n_experts, int top_k,
                               int scoring, float scale, int32_t* ids, float* weights, int n_extra, int n_pad, int n_real, float* aux,
                               int n_groups, int keep_groups, void* stream) {
  FTK_REQUIRE(groups_ok(n_experts, n_groups, keep_groups, top_k), "router_topk: %d of %d groups of %d experts, top %d", keep_groups,
              n_groups, n_experts, top_k);
  FTK_REQUIRE((n_extra == 0 || n_extra == 1) && n_pad >= 0 && n_real >= 0 && n_real <= n_experts, "router_topk: bad extra logits or expert counts");
  FTK_REQUIRE(n_parts >= 1 && n_parts <= 4, "router_topk: %d blocks of logits per token (1 to 4)", n_parts);
  FTK_REQUIRE(scoring >= FTK_SCORE_SIGMOID && scoring <= FTK_SCORE_SOFTMAX_RAW, "router_topk: unknown scoring %d", scoring);
  FTK_REQUIRE(n_experts >= 1 && top_k >= 1 && top_k <= n_experts, "router_topk: top_k=%d of %d experts", top_k, n_experts);
  FTK_REQUIRE(n_tokens >= 0, "router_topk: bad token count");
  if (n_tokens == 0) return 0;
  FTK_REQUIRE(logits && ids && weights, "router_topk: null pointer");
  const size_t smem = (size_t)kRouterWarps * 2 * n_experts * sizeof(float);
  FTK_REQUIRE(smem <= 200 * 1024, "router_topk: %d experts exceed what one block can hold (6400)", n_experts);
  if (smem > 48 * 1024) cudaFuncSetAttribute(router_topk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const int blocks = (n_tokens + kRouterWarps - 1) / kRouterWarps;
  note_variant(n_parts > 1 ? "routing: expert choice from logits given in pieces" : "routing: expert choice from given logits");
  FTK_LAUNCH(router_topk_kernel, blocks, kRouterWarps * 32, smem, (cudaStream_t)stream, logits, n_parts, bias, n_tokens, n_experts, top_k,
                                                                               scoring, scale, ids, weights, n_extra, n_pad, n_real, aux, RouteGroups{n_groups, keep_groups});
  FTK_LAUNCH_CHECK("router_topk");
  return 0;
}

static size_t route_smem(int n_tokens, int n_experts, int top_k) {
  return (size_t)(kRouteWarps * 2 + 1) * n_experts * sizeof(float) + (size_t)(n_tokens * top_k) * sizeof(int);
}

extern "C" int ftk_moe_route_fits(int n_tokens, int hidden, int n_experts, int top_k) {
  return n_tokens >= 1 && n_tokens <= 32 && hidden % 4 == 0 && n_experts >= 1 && top_k >= 1 && top_k <= n_experts &&
         route_smem(n_tokens, n_experts, top_k) <= 160 * 1024;
}

extern "C" int ftk_moe_route(const float* x, const float* gate_w, const float* bias, int n_tokens, int hidden,
                             int n_experts, int top_k, int scoring, float scale, float* logits, int32_t* ids,
                             float* weights, int32_t* counts, int32_t* offsets, int32_t* routes, int32_t* pos,
                             int do_sort, int n_extra, int n_real, float* aux, int n_groups, int keep_groups,
                             void* stream) {
  FTK_REQUIRE(groups_ok(n_experts, n_groups, keep_groups, top_k), "moe_route: %d of %d groups of %d experts, top %d", keep_groups,
              n_groups, n_experts, top_k);
  FTK_REQUIRE((n_extra == 0 || n_extra == 1) && n_real >= 0 && n_real <= n_experts, "moe_route: bad extra logits or expert counts");
  FTK_REQUIRE(scoring >= FTK_SCORE_SIGMOID && scoring <= FTK_SCORE_SOFTMAX_RAW, "moe_route: unknown scoring %d", scoring);
  FTK_REQUIRE(ftk_moe_route_fits(n_tokens, hidden, n_experts, top_k),
              "moe_route: %d tokens, width %d, %d experts, top %d do not fit the one-launch routing (at most 32 tokens, "
              "a width that is a multiple of 4); use the matrix product + router_topk + moe_permute",
              n_tokens, hidden, n_experts, top_k);
  FTK_REQUIRE(x && gate_w && logits && ids && weights, "moe_route: null pointer");
  FTK_REQUIRE(!do_sort || (counts && offsets && routes && pos), "moe_route: the sort needs its four outputs");
  FTK_REQUIRE(((uintptr_t)x | (uintptr_t)gate_w) % 16 == 0, "moe_route: x and the gate weight must be 16-byte aligned");
  const size_t smem = route_smem(n_tokens, n_experts, top_k);
  if (smem > 48 * 1024) cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const int blocks = (n_experts + n_extra + kRouteExperts - 1) / kRouteExperts;
  note_variant(do_sort ? "routing: product, choice and sort in one launch" : "routing: product and choice in one launch");
  FTK_LAUNCH(moe_route_kernel, blocks, kRouteWarps * 32, smem, (cudaStream_t)stream, 
      x, gate_w, bias, n_tokens, hidden, n_experts, top_k, scoring, scale, logits, ids, weights, counts, offsets, routes, pos,
      do_sort, n_extra, n_real, aux, RouteGroups{n_groups, keep_groups});
  FTK_LAUNCH_CHECK("moe_route");
  return 0;
}
