// Mixture of experts: softmax router, the `top` experts with the largest scores (the lower index on equal scores), their
// scores times a scale as weights, not renormalised.
//
//   route_kernel           a warp per row: scores, choice, and the row's place in each chosen expert's list
//   expert_gather_kernel   rows -> slots, one run of slots per expert, runs padded to whole tiles of 128
//   (grouped products of kernels_gemm_bf16.cuh; their sum is added by row_stats_kernel)
//   expert_token_cta       few rows: gate | up of a chosen expert as matrix-vector products
#pragma once
#include "kernels_gemm_bf16.cuh"
#include "kernels_rowwise.cuh"

namespace tg {

constexpr int MOE_LANE = 16, MOE_MAX = 32 * MOE_LANE;  // experts a warp holds
constexpr int MOE_TOP = 32;                            // most experts per token

struct MoeArgs {
	const float *z;      // [R][ldz] router logits
	int ldz, experts, top;
	float scale;
	int *id;             // [R][top]
	float *w;            // [R][top]
	int *place;          // [R][top] place in the expert's list, then the slot
	int *count;          // [experts], zero before routing
	int *tile_expert;    // [tiles]
	int *n_tiles;
	// few rows
	const float *h;      // [R][D] normed rows
	int D, n_glu;        // n_glu: activations of an expert (a multiple of 16)
	const __nv_bfloat16 *W;  // [experts][2 n_glu][ldw], blocks of 16 gate, 16 up
	int ldw, act;
	float limit;
	float *out;          // [R][top][n_glu]
};

// the warp's choice for one row; lane k < top returns the k-th (expert, weight). NL: experts per lane
template <int NL> __device__ __forceinline__ void moe_choose_n(const float *z, int E, int top, float scale, int &id, float &w) {
	const int lane = threadIdx.x & 31;
	float s[NL], mx = -INFINITY;
#pragma unroll
	for (int j = 0; j < NL; j++) {
		s[j] = lane + 32 * j < E ? z[lane + 32 * j] : -INFINITY;
		mx = fmaxf(mx, s[j]);
	}
	mx = warp_max(mx);
	float sum = 0.0f;
#pragma unroll
	for (int j = 0; j < NL; j++) {
		if (32 * j >= E) break;
		sum += expf(s[j] - mx);
	}
	sum = warp_sum(sum);
	id = 0;
	w = 0.0f;
	for (int k = 0; k < top; k++) {
		float best = -INFINITY;
		int at = 0x7fffffff;
#pragma unroll
		for (int j = 0; j < NL; j++)
			if (s[j] > best) {
				best = s[j];
				at = lane + 32 * j;
			}
#pragma unroll
		for (int x = 16; x > 0; x >>= 1) {
			const float ob = __shfl_xor_sync(0xffffffffu, best, x);
			const int oa = __shfl_xor_sync(0xffffffffu, at, x);
			if (ob > best || (ob == best && oa < at)) {
				best = ob;
				at = oa;
			}
		}
		if (at >= E) at = 0;  // (logits that are not numbers)
#pragma unroll
		for (int j = 0; j < NL; j++)
			if (lane + 32 * j == at) s[j] = -INFINITY;
		if (lane == k) {
			id = at;
			w = expf(best - mx) / sum * scale;
		}
	}
}
__device__ __forceinline__ void moe_choose(const float *z, int E, int top, float scale, int &id, float &w) {
	if (E <= 32) moe_choose_n<1>(z, E, top, scale, id, w);
	else if (E <= 128) moe_choose_n<4>(z, E, top, scale, id, w);
	else moe_choose_n<MOE_LANE>(z, E, top, scale, id, w);
}

// grid ceil(R / (8 rounds)), 256 threads, rounds <= MR_ROUNDS rows per warp. Places are counted within the CTA first: one
// addition per CTA and expert to the global counters. (A slot's number does not change what is computed there.)
constexpr int MR_ROUNDS = 8;
static __global__ void __launch_bounds__(256) route_kernel(MoeArgs a, int R, int rounds) {
	pdl_trigger();
	pdl_wait();
	__shared__ int n[MOE_MAX];
	const int lane = threadIdx.x & 31, r0 = blockIdx.x * 8 * rounds + (threadIdx.x >> 5);
	for (int e = threadIdx.x; e < a.experts; e += 256) n[e] = 0;
	__syncthreads();
	int id[MR_ROUNDS], at[MR_ROUNDS];
#pragma unroll
	for (int i = 0; i < MR_ROUNDS; i++) {
		const int r = r0 + 8 * i;
		if (i >= rounds || r >= R) break;
		float w;
		moe_choose(a.z + size_t(r) * a.ldz, a.experts, a.top, a.scale, id[i], w);
		if (lane < a.top) {
			a.id[r * a.top + lane] = id[i];
			a.w[r * a.top + lane] = w;
			at[i] = atomicAdd(n + id[i], 1);
		}
	}
	__syncthreads();
	for (int e = threadIdx.x; e < a.experts; e += 256)
		if (n[e]) n[e] = atomicAdd(a.count + e, n[e]);
	__syncthreads();
#pragma unroll
	for (int i = 0; i < MR_ROUNDS; i++) {
		const int r = r0 + 8 * i;
		if (i >= rounds || r >= R) break;
		if (lane < a.top) a.place[r * a.top + lane] = n[id[i]] + at[i];
	}
}

// grid ceil(R / rows), 128 threads, rows <= MG_ROWS: h rows of ldh (a multiple of 8) -> xg[slot]
constexpr int MG_ROWS = 4;
template <typename T> __global__ void __launch_bounds__(128) expert_gather_kernel(MoeArgs a, const T *h, int ldh, T *xg, int R, int rows) {
	pdl_trigger();
	pdl_wait();
	__shared__ int first[MOE_MAX], part[4], slot[MG_ROWS * MOE_TOP];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	// first tile of every expert: thread t owns experts 4 t .. 4 t + 3
	int c[4], sum = 0;
#pragma unroll
	for (int j = 0; j < 4; j++) {
		c[j] = 4 * tid + j < a.experts ? (a.count[4 * tid + j] + GB_BM - 1) / GB_BM : 0;
		sum += c[j];
	}
	const int r0 = blockIdx.x * rows, nr = min(rows, R - r0), items = nr * a.top;
	const int id = tid < items ? a.id[r0 * a.top + tid] : 0, place = tid < items ? a.place[r0 * a.top + tid] : 0;
	int inc = sum;
#pragma unroll
	for (int x = 1; x < 32; x *= 2) {
		const int u = __shfl_up_sync(0xffffffffu, inc, x);
		if (lane >= x) inc += u;
	}
	if (lane == 31) part[warp] = inc;
	__syncthreads();
	int at = inc - sum;
	for (int w = 0; w < warp; w++) at += part[w];
#pragma unroll
	for (int j = 0; j < 4; j++) {
		if (4 * tid + j < a.experts) first[4 * tid + j] = at;
		if (blockIdx.x == 0)
			for (int t = 0; t < c[j]; t++) a.tile_expert[at + t] = 4 * tid + j;
		at += c[j];
	}
	if (blockIdx.x == 0 && tid == 127) *a.n_tiles = at;
	__syncthreads();
	if (tid < items) {  // (MG_ROWS * MOE_TOP = 128)
		slot[tid] = first[id] * GB_BM + place;
		a.place[r0 * a.top + tid] = slot[tid];
	}
	__syncthreads();
	const int n = ldh * int(sizeof(T)) / 16;
	for (int x = tid; x < nr * n; x += 128) {
		const int i = x / n, o = x % n;
		const uint4 v = reinterpret_cast<const uint4 *>(h + size_t(r0 + i) * ldh)[o];
		for (int k = 0; k < a.top; k++) reinterpret_cast<uint4 *>(xg + size_t(slot[i * a.top + k]) * ldh)[o] = v;
	}
}

// 256 threads: 16 activations of the k-th chosen expert of row r (two per warp: 2 gate and 2 up rows). smem: h[8 ceil(D/8)]
__host__ __device__ inline int expert_token_ctas(int top, int n_glu) { return top * (n_glu / 16); }
__host__ __device__ inline size_t expert_token_smem(int D) { return size_t((D + 7) / 8 * 8) * 4; }
static __device__ void expert_token_cta(const MoeArgs &a, int r, int item, float *sm) {
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int k = item / (a.n_glu / 16), blk = item % (a.n_glu / 16), K8 = (a.D + 7) / 8;
	__shared__ int s_id;
	if (warp == 0) {
		int id;
		float w;
		moe_choose(a.z + size_t(r) * a.ldz, a.experts, a.top, a.scale, id, w);
		if (lane == k) s_id = id;
		if (item == 0 && lane < a.top) {  // (for the products that follow)
			a.id[r * a.top + lane] = id;
			a.w[r * a.top + lane] = w;
		}
	}
	for (int c = tid; c < 8 * K8; c += 256) sm[c] = c < a.D ? a.h[size_t(r) * a.D + c] : 0.0f;
	__syncthreads();
	const __nv_bfloat16 *W = a.W + (size_t(s_id) * 2 * a.n_glu + 32 * blk + 2 * warp) * a.ldw;
	float s[4] = {};
#pragma unroll 4
	for (int k8 = lane; k8 < K8; k8 += 32) {
		const float4 x0 = *reinterpret_cast<const float4 *>(sm + 8 * k8), x1 = *reinterpret_cast<const float4 *>(sm + 8 * k8 + 4);
#pragma unroll
		for (int i = 0; i < 4; i++) {
			const int4 u = ld_stream_int4(W + size_t((i >> 1) * 16 + (i & 1)) * a.ldw + 8 * k8);
			s[i] = fmaf(bf16_lo(u.x), x0.x, s[i]); s[i] = fmaf(bf16_hi(u.x), x0.y, s[i]);
			s[i] = fmaf(bf16_lo(u.y), x0.z, s[i]); s[i] = fmaf(bf16_hi(u.y), x0.w, s[i]);
			s[i] = fmaf(bf16_lo(u.z), x1.x, s[i]); s[i] = fmaf(bf16_hi(u.z), x1.y, s[i]);
			s[i] = fmaf(bf16_lo(u.w), x1.z, s[i]); s[i] = fmaf(bf16_hi(u.w), x1.w, s[i]);
		}
	}
#pragma unroll
	for (int i = 0; i < 4; i++) s[i] = warp_sum(s[i]);
	if (lane < 2) a.out[(size_t(r) * a.top + k) * a.n_glu + 16 * blk + 2 * warp + lane] = glu(a.act, a.limit, lane ? s[1] : s[0], lane ? s[3] : s[2]);
}

}  // namespace tg
