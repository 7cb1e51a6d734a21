// States and steps of the layered decoders (hybrid_model.hpp says which designs and what a layer is made of).
//
// Two pipelines compute a step; both use the same caches and states:
//   up to 4 rows, one token per sequence: matrix-vector products with the norms as prologues (kernels_gemv_bf16.cuh), five
//     launches per layer whose feed-forward follows its mixer, three where it stands beside it
//   anything else: tensor-core (or fp32) matrix products over all rows of the step
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <climits>
#include <cmath>
#include <cstdio>
#include <cstring>
#include <memory>

#include "hybrid_model.hpp"
#include "kernels_delta.cuh"
#include "kernels_gemm_bf16.cuh"
#include "kernels_gemv_bf16.cuh"
#include "kernels_moe.cuh"
#include "kernels_recurrent.cuh"
#include "kernels_rowwise.cuh"
#include "kernels_window_attn.cuh"
#include "tg_internal.hpp"

using namespace tg;

namespace {

// One token per sequence: the attention of every (sequence, key/value head, run of keys) and the delta rule of every
// (sequence, head) in one launch. grid (G * nsplit + delta heads, rows)
template <typename PT, typename CT, typename OT>
__global__ void __launch_bounds__(256) hybrid_token_mix_kernel(WAttnArgs w, DeltaArgs d) {
	pdl_trigger();
	pdl_wait();
	extern __shared__ __align__(16) float mix_sm[];
	const int n_attn = w.G * w.nsplit;
	// (the delta heads are the longer chains: they start first)
	if (int(blockIdx.x) < d.H)
		delta_token_cta<PT, OT>(d, blockIdx.y, blockIdx.x, mix_sm);
	else if (int(blockIdx.x) - d.H < n_attn)
		window_attn_token_cta<PT, CT, OT>(w, blockIdx.y, (blockIdx.x - d.H) / w.nsplit, (blockIdx.x - d.H) % w.nsplit, mix_sm);
}

// One token per sequence, the feed-forward beside the mixer: the mixer's CTAs, then (few rows) those of the row's chosen
// experts. grid (mixer CTAs + experts' CTAs, rows)
template <typename PT, typename CT, typename OT, bool ATTN, bool EXPERTS>
__global__ void __launch_bounds__(256, ATTN || EXPERTS ? 2 : 4) beside_token_mix_kernel(WAttnArgs w, LinArgs l, MoeArgs e, int n_mix) {
	pdl_trigger();
	pdl_wait();
	extern __shared__ __align__(16) float mix_sm[];
	const int x = blockIdx.x;
	if (EXPERTS && x >= n_mix) expert_token_cta(e, blockIdx.y, x - n_mix, mix_sm);
	else if (ATTN) window_attn_token_cta<PT, CT, OT>(w, blockIdx.y, x / w.nsplit, x % w.nsplit, mix_sm);
	else lin_token_cta<PT>(l, blockIdx.y, x, mix_sm);
}

// positions and history parities of the lock-step decode after a token
__global__ void hybrid_advance_kernel(int *pos, int *par, int n) {
	pdl_trigger();
	pdl_wait();
	const int i = blockIdx.x * blockDim.x + threadIdx.x;
	if (i < n) {
		pos[i] += 1;
		par[i] ^= 1;
	}
}

}  // namespace

// ===================================================================== state
struct HybridState : tg_state {
	HybridModel *m = nullptr;
	bool f32 = false;
	int max_rows = 0, max_seq_rows = 0;  // rows of a pass, rows one sequence brings to it
	struct RunCache {
		void *kc = nullptr, *vc = nullptr, *ks = nullptr, *vs = nullptr;
		int cap = 0, keep_rows = 0;
		float *canon = nullptr, *conv = nullptr, *S = nullptr, *n = nullptr, *mx = nullptr;  // n, mx: LIN_MLSTM
		CUtensorMap kmap, vmap, ksmap, vsmap;
	};
	std::vector<RunCache> cache;
	std::vector<void *> mem;
	// what a layer has computed but not yet added to x (the next norm does): its experts' outputs, partial sums
	struct Left {
		int experts = -1;  // layer
		int parts = 0;
	} left;
	float *split_part = nullptr;  // [splits][rows][ldx]
	size_t split_rows = 0;
	// activations of a pass
	float *x = nullptr;
	int ldx = 0;
	float2 *stats = nullptr;          // mean and 1/deviation of the rows
	void *h = nullptr, *hp = nullptr, *P = nullptr, *O = nullptr, *act = nullptr;  // bf16, or fp32 in a 32-bit state; hp: h before the shift
	float *T32 = nullptr;                                            // fp32 columns of the projections
	float2 *cs = nullptr;                                            // rotations of the rows' positions
	float *P32 = nullptr, *O32 = nullptr, *act32 = nullptr, *h32 = nullptr, *ex32 = nullptr;  // the few-row pipeline's, always fp32
	float *z = nullptr, *gz = nullptr, *o_raw = nullptr, *blk = nullptr, *bV = nullptr;
	void *xc = nullptr;               // convolved inputs of a recurrence
	LinArgs lin{};                    // the recurrences' buffers
	bool lin_tc = false;              // ... of the tensor-core path are there
	MoeArgs moe{};                    // routing buffers
	float *RL = nullptr;              // router logits
	void *xg = nullptr, *xa = nullptr, *xy = nullptr;  // gathered rows, experts' activations, experts' outputs
	float *part = nullptr;
	unsigned *tickets = nullptr;
	int nsplit_cap = 1;
	CUtensorMap hmap, hpmap, xgmap;   // h, hp and xg as operands
	std::vector<CUtensorMap> pmap, omap, amap, a1map, g1map, xcmap, xamap, shmap, slmap;  // per layer
	float *wl = nullptr;              // logits of wanted rows
	int wl_rows = 0;
	void *hn = nullptr;               // their normed rows
	CUtensorMap hnmap;
	int *want_dev = nullptr;
	// descriptors: of a general pass, and of the lock-step decode (row b = sequence b)
	int *desc = nullptr, *desc_pin = nullptr;
	size_t desc_ints = 0;
	int *ls_desc = nullptr, *ls_pos = nullptr, *ls_par = nullptr;
	bool ls_dirty = true;
	std::vector<int> host_par;
	// layer trace
	bool tracing = false;
	std::vector<float> trace;
	int trace_rows = 0;

	~HybridState() override {
		for (void *p : mem) cudaFree(p);
		if (desc_pin) cudaFreeHost(desc_pin);
		free_common();
	}
	int alloc();
	int reset() override;
	int prefill(const int *ids, int S, float *logits_host) override;
	int append(const int *ids, int n, float *logits_host) override;
	int enqueue_decode_all() override;
	int enqueue_forward() override;
	int run_steps(int n_steps, float minp, float temp) override;
	int step(int n, const int *seq, const int *count, const int *ids, const int *n_want, const int *want, float *logits_host) override;
	int free_sequence(int b) override;
	int trace_enable(int on) override;
	int trace_read(float *x_host, size_t cap_floats, int *runs, int *tokens) override;

	int sync_lockstep();
	StepDesc lockstep_desc() const;
	int run_layers(const StepDesc &d, int R, int nseg, int max_len);
	int score_rows(const int *rows_dev, int n, float *out, float *norm_out);
	struct GemmOpt {
		float cap = 0.0f, limit = 0.0f;
		int act = GLU_GELU, n32 = 0, ld32 = 0;
		float *C32 = nullptr;
		int splits = 0;         // GEMM_STORE32
		int bn = 0;             // columns of a tile (0: the launcher chooses)
		bool grouped = false;   // by expert: M is the most rows there can be, est the likely row tiles
		int est = 0;
	};
	int gemm(int epi, const void *A, int lda, const CUtensorMap *amap_, const Lin &w, int M, void *C, int ldc, const GemmOpt &o);
	int gemm(int epi, const void *A, int lda, const CUtensorMap *amap_, const Lin &w, int M, void *C, int ldc) { return gemm(epi, A, lda, amap_, w, M, C, ldc, GemmOpt()); }
	int gemv(int pro, int epi, GemvArgs g, int R);
	WAttnArgs attn_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo);
	DeltaArgs delta_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo);
	LinArgs lin_args(const StepDesc &d, int run, const void *p);
	MoeArgs moe_args(const Layer &L);
	int moe_rows(const Layer &L, int rows) const { return (rows * L.ff.top / GB_BM + L.ff.experts) * GB_BM; }
	int few_layer(const StepDesc &d, int run, int R);
	int rows_layer(const StepDesc &d, int run, int R, int nseg, int max_len);
	int beside_few_layer(const StepDesc &d, int run, int R);
	int beside_rows_layer(const StepDesc &d, int run, int R, int nseg, int max_len);
	int norm_in(const StepDesc &d, int run, int R);  // what is left is added; norm1 and what follows it
	int add_left(int R);
	template <typename T> RowSum<T> row_sum(int R);
	int attn_rows(const WAttnArgs &wa, int run, int R, int nseg, int max_len);
	int token_splits(const WAttnArgs &wa, int fill) const;
	int few_rows() const;

	struct Entry {
		int seq, count, done;
		const int *ids;
		std::vector<int> want;  // places
		size_t out0;            // first output row
		size_t given = 0;       // wanted rows already scored
	};
	// last = true: instead of `want`, the last token of every entry is scored into `logits` (row = sequence)
	int run_entries(std::vector<Entry> &es, bool last, float *logits_host);

	template <typename T> int take(T **p, size_t n) {
		if (n == 0) n = 1;
		cudaError_t e = cudaMalloc(reinterpret_cast<void **>(p), n * sizeof(T));
		if (e != cudaSuccess) {
			cudaGetLastError();
			return fail(TG_ENOMEM, std::string("cudaMalloc(state): ") + cudaGetErrorString(e));
		}
		mem.push_back(*p);
		TG_CUDA(cudaMemsetAsync(*p, 0, n * sizeof(T), stream));
		return TG_OK;
	}
	int take_act(void **p, size_t n) {
		uint8_t *q;
		TG_TRY(take(&q, n * (f32 ? 4 : 2)));
		*p = q;
		return TG_OK;
	}
};

namespace {
constexpr int FEW_ROWS = 4;  // rows of the matrix-vector pipeline
constexpr int TOKEN_SPLITS = 32;
constexpr int LIN_SCAN_MAX = 8;  // portions up to this long go through a recurrence token by token

template <typename K> int allow_smem(K kernel, size_t bytes) {
	if (bytes <= 48 * 1024) return TG_OK;
	if (bytes > 227 * 1024) return fail(TG_ESHAPE, "a layer's sizes need more shared memory than an SM has");
	TG_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(bytes)));
	return TG_OK;
}

// columns of a tile: waves x measured time of a K-block (a tile is bound by what it reads from the L2)
int pick_bn(int m_tiles, int N) {
	static const int forced = env_int("TG_GEMM_BN", 0);
	if (forced) return forced;
	int best = 64;
	double cost = 1e30;
	for (int bn : {256, 128, 64}) {
		const int tiles = m_tiles * ((N + bn - 1) / bn);
		const double c = double((tiles + g_num_sms - 1) / g_num_sms) * (bn == 256 ? 1.0 : (bn == 128 ? 0.79 : 0.6));
		if (c < cost) {
			cost = c;
			best = bn;
		}
	}
	return best;
}

// The same for a product whose K several CTAs may share, their partial sums being added later: what a tile costs is its
// K-blocks and a fixed part, and a partial sum is written and read once more.
void pick_split(int M, int N, int K, int *bn, int *splits) {
	static const int most = env_int("TG_SPLIT_K", 8);
	const int m_tiles = (M + GB_BM - 1) / GB_BM, kb = (K + GB_BK - 1) / GB_BK;
	double best = 1e30;
	for (int b : {256, 128, 64})
		for (int s = 1; s <= std::min(most, std::max(1, kb / 4)); s++) {
			if ((s - 1) * ((kb + s - 1) / s) >= kb) continue;  // (every share has work)
			const int tiles = m_tiles * ((N + b - 1) / b) * s;
			const double c = double((tiles + g_num_sms - 1) / g_num_sms) * ((kb + s - 1) / s + 4) * (b == 256 ? 0.35 : (b == 128 ? 0.275 : 0.21))  // us
			                 + (s > 1 ? 1.0 + s * double(M) * N * 8.0 / 6e6 : 0.0);
			if (c < best) {
				best = c;
				*bn = b;
				*splits = s;
			}
		}
}

template <int BN, int EPI, bool GRP> int launch_gemm_tc(const CUtensorMap &am, const CUtensorMap &wm, const GemmArgs &a, cudaStream_t st) {
	static bool done[TG_MAX_DEVICES] = {};
	bool &d = done[current_device_slot()];
	auto kernel = gemm_bf16_tc_kernel<BN, EPI, GRP>;
	if (!d) {
		TG_TRY(allow_smem(kernel, GbShape<BN>::SMEM));
		d = true;
	}
	launch_k(kernel, dim3(std::min(g_num_sms, a.m_tiles * a.n_tiles * std::max(1, a.splits))), dim3(GB_THREADS), size_t(GbShape<BN>::SMEM), st, am, wm, a);
	count_launch();
	return check_launch("gemm_bf16_tc");
}
// est: row tiles that a grouped product is likely to have
template <int EPI, bool GRP = false> int launch_gemm(const CUtensorMap &am, const Lin &w, GemmArgs a, cudaStream_t st, int est = 0, int want_bn = 0) {
	a.m_tiles = (a.M + GB_BM - 1) / GB_BM;
	const int cols = EPI == GEMM_LOGITS ? a.ldc : a.N, bn = want_bn ? want_bn : pick_bn(est ? est : a.m_tiles, cols);
	a.n_tiles = (cols + bn - 1) / bn;
	if (bn == 256) return launch_gemm_tc<256, EPI, GRP>(am, w.map[2], a, st);
	if (bn == 128) return launch_gemm_tc<128, EPI, GRP>(am, w.map[1], a, st);
	return launch_gemm_tc<64, EPI, GRP>(am, w.map[0], a, st);
}
template <int EPI, bool GRP = false> int launch_gemm_f32(const float *A, int lda, const Lin &w, const GemmArgs &a, cudaStream_t st) {
	const int cols = EPI == GEMM_LOGITS ? a.ldc : a.N;
	launch_k(gemm_f32_kernel<EPI, GRP>, dim3((cols + GF_T - 1) / GF_T, (a.M + GF_T - 1) / GF_T), dim3(256), 0, st, A, lda, w.W, w.ld, a);
	count_launch();
	return check_launch("gemm_f32");
}

template <int R, int NR, int KS, int PRO, int EPI> int launch_gemv(const GemvArgs &g, cudaStream_t st) {
	const size_t smem = gv_smem<R, NR>(g.K, PRO, EPI, g.parts, g.top, g.top * g.n_ex);
	auto kernel = gemv_bf16_kernel<R, NR, KS, PRO, EPI>;
	TG_TRY(allow_smem(kernel, smem));
	int occ = 1;
	TG_CUDA(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, kernel, GV_THREADS, smem));
	const int outs = (8 / KS) * NR / (EPI == GV_GLU ? 2 : 1);
	const int n_out = EPI == GV_GLU ? g.N / 2 : (EPI == GV_LOGITS ? g.ldo : g.N);
	auto per = [](int n, int m) { return (n + m - 1) / m; };
	const int groups = EPI == GV_FRONT ? per(g.n_proj, outs) + per(g.n_glu, outs / 2) + per(g.n_route, outs) : per(n_out, outs);
	launch_k(kernel, dim3(std::min(groups, std::max(1, occ) * g_num_sms)), dim3(GV_THREADS), smem, st, g);
	count_launch();
	return check_launch("gemv_bf16");
}
template <int R> int launch_gemv_r(int pro, int epi, const GemvArgs &g, cudaStream_t st) {
	if (pro == GV_LN_CONV && epi == GV_PROJ) return launch_gemv<R, 4, 2, GV_LN_CONV, GV_PROJ>(g, st);
	if (pro == GV_VEC && epi == GV_ADD) return launch_gemv<R, 4, 8, GV_VEC, GV_ADD>(g, st);
	if (pro == GV_LN && epi == GV_GLU) return launch_gemv<R, 4, 2, GV_LN, GV_GLU>(g, st);
	if (pro == GV_LN_CONV && epi == GV_FRONT) return launch_gemv<R, 4, 2, GV_LN_CONV, GV_FRONT>(g, st);
	if (pro == GV_MIX && epi == GV_ADD) return launch_gemv<R, 4, 8, GV_MIX, GV_ADD>(g, st);
	if (pro == GV_LN && epi == GV_LOGITS) return launch_gemv<R, 4, 2, GV_LN, GV_LOGITS>(g, st);
	return fail(TG_EINVAL, "gemv: no such combination");
}
}  // namespace

int HybridModel::new_state(int batch, int max_pos, tg_state **out) {
	HybridState *s = new HybridState();
	s->m = this;
	s->model = this;
	s->B = batch;
	s->max_pos_global = max_pos;
	s->f32 = dtype == TG_F32;
	const int rc = s->alloc();
	if (rc != TG_OK) {
		const std::string keep = tg_last_error();
		tg_state_free(s);
		return fail(rc, keep);
	}
	*out = s;
	return TG_OK;
}

int HybridState::alloc() {
	TG_TRY(alloc_common());
	const int D = m->D;
	const int pass = std::max(B, env_int("TG_PASS_ROWS", 4096));
	max_seq_rows = std::min(std::max(128, pass / B), max_pos_global);
	max_rows = std::min<long long>(std::max(pass, B), (long long)B * max_seq_rows);
	const int R = max_rows;
	const size_t es = f32 ? 4 : 2;
	ldx = round_up(D, 8);
	int ldp = 8, kc = 8, ffp = 16, hz = 1, hv = 1, tail = 0, xcn = 0, inner = 0, half = m->rot_half;
	size_t blkn = 0, blkV = 0, partn = 1;
	int gmax = 1;
	bool beside = false;
	size_t linS = 0, linSp = 0, linN = 0;  // per chunk: state rows x columns (two paddings), key vectors
	int linH = 0, top = 0, experts = 0, slots = 0, effp = 0, exf = 0;
	for (const Layer &L : m->layers) {
		ldp = std::max(ldp, L.ldp);
		kc = std::max(kc, L.kcat);
		ffp = std::max(ffp, L.ff.ffp);
		tail = std::max(tail, L.tail());
		beside = beside || L.beside;
		if (L.de.H) {
			hz = std::max(hz, round_up(L.de.H * L.de.dk, 4));
			hv = std::max(hv, round_up(L.de.H * L.de.dv, 4));
			blkn = std::max(blkn, size_t(L.de.H) * delta_block_floats(L.de.dkp()));
			blkV = std::max(blkV, size_t(L.de.H) * DB * L.de.dv);
		}
		if (L.at.H) {
			partn = std::max(partn, size_t(L.at.H) * (L.at.dvp + 2));
			gmax = std::max(gmax, L.at.G);
		}
		if (L.li.H) {
			const LinSpec &li = L.li;
			inner = std::max(inner, round_up(li.H * li.vd, 4));
			linH = std::max(linH, li.H);
			if (li.kind == LIN_SSM) xcn = std::max(xcn, li.xc_cols());
			if (li.Np <= 256) {
				linS = std::max(linS, size_t(li.H) * li.N * li.vdp);
				linSp = std::max(linSp, size_t(li.H) * li.Np * li.vdp);
				linN = std::max(linN, size_t(li.H) * li.N);
			}
		}
		if (L.ff.experts) {
			top = std::max(top, L.ff.top);
			experts = std::max(experts, round_up(L.ff.experts, 8));
			slots = std::max(slots, moe_rows(L, R));
			effp = std::max(effp, L.ff.effp);
			exf = std::max(exf, L.ff.top * L.ff.effp);
		}
	}
	TG_TRY(take(&x, size_t(R) * ldx));
	TG_TRY(take(&stats, R));
	TG_TRY(take_act(&h, size_t(R) * m->Dp));
	TG_TRY(take_act(&P, size_t(R) * ldp));
	TG_TRY(take_act(&O, size_t(R) * kc));
	if (beside) TG_TRY(take_act(&hp, size_t(R) * m->Dp));
	else TG_TRY(take_act(&act, size_t(R) * ffp));
	TG_TRY(take(&T32, size_t(R) * tail));
	if (half) TG_TRY(take(&cs, size_t(R) * m->rots.size() * half));
	const int F = std::min(FEW_ROWS, B);
	TG_TRY(take(&P32, size_t(F) * ldp));
	TG_TRY(take(&O32, size_t(F) * kc));
	TG_TRY(take(&act32, size_t(F) * ffp));
	TG_TRY(take(&h32, size_t(F) * D));
	TG_TRY(take(&ex32, size_t(F) * exf));
	TG_TRY(take(&o_raw, size_t(R) * std::max(hv, inner)));
	if (blkn) {
		TG_TRY(take(&z, size_t(R) * hz));
		TG_TRY(take(&gz, size_t(R) * hv));
		const size_t nb = size_t(R) / DB + B + 1;
		TG_TRY(take(&blk, nb * blkn));
		TG_TRY(take(&bV, nb * blkV));
	}
	if (beside && !f32) {
		split_rows = std::min(size_t(8) * R, size_t(4096));
		TG_TRY(take(&split_part, split_rows * ldx));
	}
	if (linH) {
		if (xcn) TG_TRY(take_act(&xc, size_t(R) * xcn));
		TG_TRY(take(&lin.la, size_t(R) * linH));
		TG_TRY(take(&lin.b, size_t(R) * linH));
		TG_TRY(take(&lin.em, size_t(R) * linH));
	}
	const size_t nchunk = size_t(R) / LC + B + 1;
	lin_tc = !f32 && linS && env_int("TG_LIN_TC", 1);
	if (lin_tc) {
		TG_TRY(take(&lin.dS, nchunk * linS));
		TG_TRY(take(&lin.Sh, nchunk * linSp));
		TG_TRY(take(&lin.Sl, nchunk * linSp));
		TG_TRY(take(&lin.dn, nchunk * linN));
		TG_TRY(take(&lin.n0, nchunk * linN));
		TG_TRY(take(&lin.tot, nchunk * linH));
	}
	if (experts) {
		TG_TRY(take(&RL, size_t(R) * experts));
		TG_TRY(take(&moe.id, size_t(R) * top));
		TG_TRY(take(&moe.w, size_t(R) * top));
		TG_TRY(take(&moe.place, size_t(R) * top));
		TG_TRY(take(&moe.count, experts));
		TG_TRY(take(&moe.tile_expert, slots / GB_BM));
		TG_TRY(take(&moe.n_tiles, 1));
		TG_TRY(take_act(&xg, size_t(slots) * m->Dp));
		TG_TRY(take_act(&xa, size_t(slots) * effp));
		TG_TRY(take_act(&xy, size_t(slots) * ldx));
	}
	nsplit_cap = std::max(1, std::min(TOKEN_SPLITS, 2 * g_num_sms / B));
	TG_TRY(take(&part, size_t(B) * nsplit_cap * partn));
	TG_TRY(take(&tickets, size_t(B) * gmax));
	// caches
	cache.resize(m->runs.size());
	for (size_t i = 0; i < cache.size(); i++) {
		const Layer &L = m->layers[m->runs[i].layer];
		const AttnSpec &A = L.at;
		RunCache &c = cache[i];
		if (m->taps > 1) TG_TRY(take(&c.canon, size_t(B) * 2 * (m->taps - 1) * D));
		if (L.de.H) {
			TG_TRY(take(&c.conv, size_t(B) * 2 * (L.de.taps - 1) * L.de.channels()));
			TG_TRY(take(&c.S, size_t(B) * L.de.H * L.de.dk * L.de.dv));
		}
		if (L.li.H) {
			TG_TRY(take(&c.S, size_t(B) * L.li.H * L.li.N * L.li.vdp));
			if (L.li.kind == LIN_SSM) {
				TG_TRY(take(&c.conv, size_t(B) * 2 * (L.li.taps - 1) * L.li.channels()));
			} else {
				TG_TRY(take(&c.n, size_t(B) * 2 * L.li.H * L.li.N));
				TG_TRY(take(&c.mx, size_t(B) * 2 * L.li.H));
			}
		}
		if (!A.H) continue;
		// (a pooled block is formed from the ring, so the ring reaches back a whole block)
		c.cap = round_up(int(std::min<long long>(max_pos_global, (long long)std::max(A.window, A.pool) + max_seq_rows)), 64);
		c.keep_rows = round_up(A.pool ? max_pos_global / A.pool : std::min(A.keep, max_pos_global), 64);
		uint8_t *q;
		auto rows = [&](void **p, size_t n, int w) -> int {
			TG_TRY(take(&q, size_t(B) * n * w * es));
			*p = q;
			return TG_OK;
		};
		TG_TRY(rows(&c.kc, c.cap, A.G * A.dkp));
		TG_TRY(rows(&c.vc, c.cap, A.G * A.dvp));
		TG_TRY(rows(&c.ks, c.keep_rows, A.G * A.dkp));
		TG_TRY(rows(&c.vs, c.keep_rows, A.G * A.dvp));
		if (!f32) {
			TG_TRY(make_map(&c.kmap, c.kc, size_t(B) * c.cap, A.G * A.dkp, A.G * A.dkp, WT_KEYS));
			TG_TRY(make_map(&c.vmap, c.vc, size_t(B) * c.cap, A.G * A.dvp, A.G * A.dvp, WT_KEYS));
			c.ksmap = c.kmap;  // (not used without a second store)
			c.vsmap = c.vmap;
			if (c.keep_rows) {
				TG_TRY(make_map(&c.ksmap, c.ks, size_t(B) * c.keep_rows, A.G * A.dkp, A.G * A.dkp, WT_KEYS));
				TG_TRY(make_map(&c.vsmap, c.vs, size_t(B) * c.keep_rows, A.G * A.dvp, A.G * A.dvp, WT_KEYS));
			}
		}
	}
	// wanted rows
	wl_rows = std::max(16, std::min(1024, int((size_t(64) << 20) / ld_logits)));
	wl_rows = std::min(wl_rows, std::max(16, R));
	TG_TRY(take(&wl, size_t(wl_rows) * ld_logits));
	TG_TRY(take_act(&hn, size_t(std::max(wl_rows, B)) * m->Dp));
	TG_TRY(take(&want_dev, wl_rows));
	if (!f32) {
		TG_TRY(make_map(&hmap, h, R, m->Dp, m->Dp, GB_BM));
		TG_TRY(make_map(&hnmap, hn, std::max(wl_rows, B), m->Dp, m->Dp, GB_BM));
		const size_t n = m->layers.size();
		if (beside) TG_TRY(make_map(&hpmap, hp, R, m->Dp, m->Dp, GB_BM));
		if (experts) TG_TRY(make_map(&xgmap, xg, slots, m->Dp, m->Dp, GB_BM));
		for (auto *v : {&pmap, &omap, &amap, &a1map, &g1map, &xcmap, &xamap, &shmap, &slmap}) v->resize(n);
		for (size_t i = 0; i < n; i++) {
			const Layer &L = m->layers[i];
			const bf16 *p = static_cast<const bf16 *>(P);
			TG_TRY(make_map(&pmap[i], P, R, L.ldp, L.ldp, 128));
			TG_TRY(make_map(&omap[i], O, R, L.kcat, L.kcat, GB_BM));
			if (!L.beside && L.ff.ff) TG_TRY(make_map(&amap[i], act, R, L.ff.ffp, L.ff.ffp, GB_BM));
			if (L.de.H) {
				TG_TRY(make_map(&a1map[i], p + L.p_a1, R, L.de.ra, L.ldp, GB_BM));
				TG_TRY(make_map(&g1map[i], p + L.p_g1, R, L.de.rg, L.ldp, GB_BM));
			}
			const LinSpec &li = L.li;
			if (li.kind == LIN_SSM) TG_TRY(make_map(&xcmap[i], xc, R, li.xc_cols(), li.xc_cols(), LC));
			if (lin_tc && li.H && li.Np <= 256) {
				TG_TRY(make_map(&shmap[i], lin.Sh, nchunk * li.H * li.Np, li.vdp, li.vdp, li.Np));
				TG_TRY(make_map(&slmap[i], lin.Sl, nchunk * li.H * li.Np, li.vdp, li.vdp, li.Np));
			}
			if (L.ff.experts) TG_TRY(make_map(&xamap[i], xa, moe_rows(L, R), L.ff.effp, L.ff.effp, GB_BM));
		}
	}
	// descriptors
	desc_ints = size_t(2) * R + 5 * size_t(B);
	TG_TRY(take(&desc, desc_ints));
	TG_CUDA(cudaMallocHost(&desc_pin, desc_ints * 4));
	TG_TRY(take(&ls_desc, size_t(5) * B));
	ls_pos = ls_desc + 3 * B;
	ls_par = ls_desc + 4 * B;
	std::vector<int> init(size_t(5) * B, 0);
	for (int b = 0; b < B; b++) {
		init[b] = b;          // row -> segment, segment -> sequence, segment -> first row
		init[B + b] = 1;      // length
	}
	TG_CUDA(cudaMemcpyAsync(ls_desc, init.data(), init.size() * 4, cudaMemcpyHostToDevice, stream));
	host_par.assign(B, 0);
	TG_CUDA(cudaStreamSynchronize(stream));
	return TG_OK;
}

StepDesc HybridState::lockstep_desc() const {
	StepDesc d;
	d.tok = tok;
	d.row_seg = d.seg_seq = d.seg_row = ls_desc;
	d.seg_len = ls_desc + B;
	d.seg_pos = ls_pos;
	d.seg_par = ls_par;
	return d;
}

// the device's positions and parities of the lock-step decode follow the host's after anything else has run
int HybridState::sync_lockstep() {
	if (!ls_dirty) return TG_OK;
	TG_CUDA(cudaStreamSynchronize(stream));  // (desc_pin may still be read by an earlier copy)
	for (int b = 0; b < B; b++) {
		desc_pin[b] = host_pos[b];
		desc_pin[B + b] = host_par[b];
	}
	TG_CUDA(cudaMemcpyAsync(ls_pos, desc_pin, size_t(2) * B * 4, cudaMemcpyHostToDevice, stream));
	ls_dirty = false;
	return TG_OK;
}

int HybridState::reset() {
	// What caches and histories hold is never read before it has been written again: rows at negative positions count
	// as zero, and a state matrix is read from position 1 on.
	host_par.assign(B, 0);
	ls_dirty = true;
	return TG_OK;
}

int HybridState::free_sequence(int b) {
	TG_CUDA(cudaStreamSynchronize(stream));
	host_pos[b] = 0;
	host_par[b] = 0;
	ls_dirty = true;
	return TG_OK;
}

int HybridState::trace_enable(int on) {
	tracing = on != 0;
	trace.clear();
	trace_rows = 0;
	return TG_OK;
}

int HybridState::trace_read(float *x_host, size_t cap_floats, int *runs, int *tokens) {
	*runs = trace_rows ? int(m->runs.size()) : 0;
	*tokens = trace_rows;
	if (!x_host) return TG_OK;
	if (cap_floats < trace.size()) return fail(TG_EINVAL, "buffer too small for the trace");
	std::memcpy(x_host, trace.data(), trace.size() * 4);
	return TG_OK;
}

// ------------------------------------------------------------------ pieces of a step
int HybridState::gemm(int epi, const void *A, int lda, const CUtensorMap *am, const Lin &w, int M, void *C, int ldc, const GemmOpt &o) {
	GemmArgs a{};
	a.M = M;
	a.N = w.N;
	a.K = w.K;
	a.C = C;
	a.ldc = ldc;
	a.cap = o.cap;
	a.err = err_flag;
	a.act = o.act;
	a.limit = o.limit;
	a.n32 = o.n32;
	a.C32 = o.C32;
	a.ld32 = o.ld32;
	a.tile_expert = moe.tile_expert;
	a.n_row_tiles = moe.n_tiles;
	a.splits = o.splits;
	if (f32) {
		const float *Af = static_cast<const float *>(A);
		switch (epi) {
			case GEMM_ADD: return launch_gemm_f32<GEMM_ADD>(Af, lda, w, a, stream);
			case GEMM_GLU: return o.grouped ? launch_gemm_f32<GEMM_GLU, true>(Af, lda, w, a, stream) : launch_gemm_f32<GEMM_GLU>(Af, lda, w, a, stream);
			case GEMM_LOGITS: return launch_gemm_f32<GEMM_LOGITS>(Af, lda, w, a, stream);
			default: return o.grouped ? launch_gemm_f32<GEMM_STORE, true>(Af, lda, w, a, stream) : launch_gemm_f32<GEMM_STORE>(Af, lda, w, a, stream);
		}
	}
	if (o.grouped) return epi == GEMM_GLU ? launch_gemm<GEMM_GLU, true>(*am, w, a, stream, o.est) : launch_gemm<GEMM_STORE, true>(*am, w, a, stream, o.est);
	switch (epi) {
		case GEMM_STORE: return launch_gemm<GEMM_STORE>(*am, w, a, stream);
		case GEMM_STORE32: return launch_gemm<GEMM_STORE32>(*am, w, a, stream, 0, o.bn);
		case GEMM_ADD: return launch_gemm<GEMM_ADD>(*am, w, a, stream);
		case GEMM_GLU: return launch_gemm<GEMM_GLU>(*am, w, a, stream);
		default: return launch_gemm<GEMM_LOGITS>(*am, w, a, stream);
	}
}

int HybridState::gemv(int pro, int epi, GemvArgs g, int R) {
	g.err = err_flag;
	g.rms = m->rms;
	g.embed_scale = m->embed_scale;
	// (rows whose activations do not fit shared memory together go in smaller groups)
	int most = R >= 4 ? 4 : (R >= 2 ? 2 : 1);
	const size_t row_floats = size_t(epi == GV_FRONT ? 3 : (pro == GV_LN_CONV ? 2 : 1)) * 8 * gv_k8(g.K) + (pro == GV_MIX ? g.top * g.n_ex : 0);
	while (most > 1 && most * row_floats * 4 > 160 * 1024) most /= 2;
	for (int r = 0; r < R;) {
		int n = most;
		while (n > R - r) n /= 2;
		GemvArgs s = g;
		s.d.tok += r;
		s.d.row_seg += r;
		if (s.vec) s.vec += size_t(r) * g.ldv;
		if (s.x) s.x += size_t(r) * g.ldx;
		s.out += size_t(r) * g.ldo;
		if (s.out32) s.out32 += size_t(r) * g.ld32;
		if (s.glu_out) s.glu_out += size_t(r) * g.ld_glu;
		if (s.route_out) s.route_out += size_t(r) * g.ld_route;
		if (s.gate) s.gate += size_t(r) * g.ldg;
		if (s.top) {
			s.ex_act += size_t(r) * g.top * g.n_ex;
			s.ex_w += r * g.top;
			s.ex_id += r * g.top;
		}
		if (s.norm_out) s.norm_out += size_t(r) * g.D;
		TG_TRY(n == 4 ? launch_gemv_r<4>(pro, epi, s, stream) : (n == 2 ? launch_gemv_r<2>(pro, epi, s, stream) : launch_gemv_r<1>(pro, epi, s, stream)));
		r += n;
	}
	return TG_OK;
}

WAttnArgs HybridState::attn_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo) {
	const Layer &L = m->layers[m->runs[run].layer];
	const RunCache &c = cache[run];
	WAttnArgs a{};
	a.d = d;
	a.H = L.at.H;
	a.G = L.at.G;
	a.dk = L.at.dk;
	a.dv = L.at.dv;
	a.dkp = L.at.dkp;
	a.dvp = L.at.dvp;
	a.scale = L.at.scale;
	a.window = L.at.window;
	a.keep = std::min(L.at.keep, c.keep_rows);
	a.pool = L.at.pool;
	if (L.at.rot >= 0) {
		a.rot = L.at.rot_dims;
		a.cs = cs + size_t(L.at.rot) * max_rows * m->rot_half;
		a.ld_cs = m->rot_half;
	}
	a.vnorm = L.at.vnorm;
	a.eps = m->eps;
	a.r1 = L.r1;
	a.r2 = L.r2;
	a.p = p;
	a.ldp = ldp;
	a.p_q = L.p_q;
	a.p_k = L.p_k;
	a.p_v = L.p_v;
	a.p_g = L.at.gated ? L.p_g : -1;
	a.kc = c.kc;
	a.vc = c.vc;
	a.ks = c.ks;
	a.vs = c.vs;
	a.cap = c.cap;
	a.keep_rows = c.keep_rows;
	a.out = out;
	a.ldo = ldo;
	a.out_scale = L.left_scale;
	a.part = part;
	a.tickets = tickets;
	a.nsplit = 1;
	a.err = err_flag;
	return a;
}

DeltaArgs HybridState::delta_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo) {
	const Layer &L = m->layers[m->runs[run].layer];
	const RunCache &c = cache[run];
	DeltaArgs a{};
	a.d = d;
	a.H = L.de.H;
	a.KH = L.de.KH;
	a.dk = L.de.dk;
	a.dv = L.de.dv;
	a.taps = L.de.taps;
	a.p = p;
	a.ldp = ldp;
	a.p_conv = L.p_conv;
	a.p_b = L.p_b;
	a.cw = L.conv;
	a.hist = c.conv;
	a.A_log = L.A_log;
	a.dt_bias = L.dt_bias;
	a.z = z;
	a.gz = gz;
	a.ldz = round_up(L.de.H * L.de.dk, 4);
	a.ldgz = round_up(L.de.H * L.de.dv, 4);
	a.S = c.S;
	a.norm = L.rnorm;
	a.eps = m->eps;
	a.out_scale = L.right_scale;
	a.out = out;
	a.ldo = ldo;
	a.o_col = L.o_col;
	a.ra = L.de.ra;
	a.rg = L.de.rg;
	a.p_a1 = L.p_a1;
	a.p_g1 = L.p_g1;
	a.a2 = L.a2.W;
	a.g2 = L.g2.W;
	a.lda2 = L.a2.ld;
	a.ldg2 = L.g2.ld;
	a.dkp = L.de.dkp();
	a.blk = blk;
	a.bV = bV;
	a.err = err_flag;
	a.o = o_raw;
	return a;
}

// p: projections of the rows
LinArgs HybridState::lin_args(const StepDesc &d, int run, const void *p) {
	const Layer &L = m->layers[m->runs[run].layer];
	const LinSpec &s = L.li;
	const RunCache &c = cache[run];
	LinArgs a = lin;
	a.d = d;
	a.kind = s.kind;
	a.H = s.H;
	a.G = s.G;
	a.N = s.N;
	a.vd = s.vd;
	a.Np = s.Np;
	a.vdp = s.vdp;
	a.p = p;
	a.ldp = L.ldp;
	a.p_x = L.p_conv;
	a.p_q = L.p_q;
	a.p_k = L.p_k;
	a.p_v = L.p_v;
	a.t = T32;
	a.ldt = L.tail();
	a.A_log = L.A_log;
	a.dt_bias = L.dt_bias;
	a.Dv = L.Dv;
	a.ib = L.ib;
	a.fb = L.fb;
	a.gate_cap = s.gate_cap;
	a.qscale = s.kind == LIN_MLSTM ? 1.0f / std::sqrt(float(s.N)) : 1.0f;
	a.cw = L.conv;
	a.cb = L.conv_b;
	a.taps = s.taps;
	a.hist = c.conv;
	a.xc = xc;
	a.ldxc = s.xc_cols();
	if (s.kind == LIN_SSM) {
		a.rows = xc;
		a.ldr = a.ldxc;
		a.o_v = 0;
		a.o_k = s.H * s.vdp;
		a.o_q = a.o_k + s.G * s.Np;
	} else {
		a.rows = p;
		a.ldr = L.ldp;
		a.o_q = L.p_q;
		a.o_k = L.p_k;
		a.o_v = L.p_v;
	}
	a.S = c.S;
	a.n = c.n;
	a.m = c.mx;
	a.o = o_raw;
	a.ldo = round_up(s.H * s.vd, 4);
	a.vsplit = 1;
	a.err = err_flag;
	return a;
}

MoeArgs HybridState::moe_args(const Layer &L) {
	MoeArgs a = moe;
	a.z = RL;
	a.ldz = round_up(L.ff.experts, 8);
	a.experts = L.ff.experts;
	a.top = L.ff.top;
	a.scale = L.ff.route_scale;
	a.h = h32;
	a.D = m->D;
	a.n_glu = L.ff.effp;
	a.W = L.ex_gu.W;
	a.ldw = L.ex_gu.ld;
	a.act = L.ff.act;
	a.limit = L.ff.limit;
	a.out = ex32;
	return a;
}

namespace {
template <typename PT, typename CT, typename OT> int launch_token_mix(const WAttnArgs &w, const DeltaArgs &d, int R, cudaStream_t st) {
	const size_t smem = std::max(wattn_token_smem(w.H / w.G, w.dkp, w.dvp), delta_token_smem(d.dk, d.dv, d.ra, d.rg));
	auto kernel = hybrid_token_mix_kernel<PT, CT, OT>;
	TG_TRY(allow_smem(kernel, smem));
	launch_k(kernel, dim3(w.G * w.nsplit + d.H, R), dim3(256), smem, st, w, d);
	count_launch();
	return check_launch("hybrid_token_mix");
}
template <int RPL, int NW, int NC> int launch_scan_nc(const DeltaArgs &a, int nseg, cudaStream_t st) {
	const int groups = (a.dv + 4 * NC - 1) / (4 * NC);
	// few CTAs: deep prefetch; many: more of them per SM
	int stages = (long long)groups * a.H * nseg <= 2 * g_num_sms ? 4 : 2;
	while (stages > 2 && delta_scan_smem<RPL, NW, NC>(stages) > 200 * 1024) stages--;
	const size_t smem = delta_scan_smem<RPL, NW, NC>(stages);
	auto kernel = delta_scan_kernel<RPL, NW, NC>;
	TG_TRY(allow_smem(kernel, smem));
	launch_k(kernel, dim3(groups, a.H, nseg), dim3(32 * NW), smem, st, a, stages);
	count_launch();
	return check_launch("delta_scan");
}
// columns per lane: one while every SM gets at most one CTA, more (fewer shared-memory reads per column) beyond
template <int RPL, int NW> int launch_scan(const DeltaArgs &a, int nseg, cudaStream_t st) {
	static const int forced = env_int("TG_SCAN_COLS", 0);
	const long long cols = (long long)a.dv * a.H * nseg;
	const int nc = forced ? forced : (cols <= 4 * g_num_sms ? 1 : (cols <= 40 * g_num_sms ? 2 : 4));
	if (nc == 1) return launch_scan_nc<RPL, NW, 1>(a, nseg, st);
	if (nc == 2) return launch_scan_nc<RPL, NW, 2>(a, nseg, st);
	return launch_scan_nc<RPL, NW, 4>(a, nseg, st);
}
template <typename PT> int launch_delta(const DeltaArgs &a, int R, int nseg, int max_len, cudaStream_t st) {
	const size_t smem = delta_block_smem(a.dkp, a.dv);
	TG_TRY(allow_smem(delta_block_kernel<PT>, smem));
	launch_k(delta_block_kernel<PT>, dim3((max_len + DB - 1) / DB, a.H, nseg), dim3(256), smem, st, a);
	count_launch();
	TG_TRY(check_launch("delta_block"));
	switch (a.dkp) {
		case 32: TG_TRY((launch_scan<4, 1>(a, nseg, st))); break;
		case 64: TG_TRY((launch_scan<4, 2>(a, nseg, st))); break;
		case 128: TG_TRY((launch_scan<4, 4>(a, nseg, st))); break;
		default: TG_TRY((launch_scan<8, 4>(a, nseg, st))); break;
	}
	launch_k(delta_out_kernel<PT>, dim3((R * a.H + 7) / 8), dim3(256), 0, st, a, R);
	count_launch();
	return check_launch("delta_out");
}
template <typename PT> int launch_stats(float2 *stats, float *x, int ldx, int R, int D, float eps, int rms, const RowSum<PT> &add, cudaStream_t st) {
	launch_k(row_stats_kernel<PT>, dim3(R), dim3(128), 0, st, stats, x, ldx, D, eps, rms, add);
	count_launch();
	return check_launch("row_stats");
}
template <typename PT> int launch_norm_conv(void *out, void *plain, int ldo, const float *x, int ldx, const float2 *stats, const float *w, const float *cw, float *hist,
                                            const StepDesc &d, int R, int D, int taps, cudaStream_t st) {
	const int cols = (ldo + 511) / 512;
	int rows = LC_ROWS;
	while (rows > 1 && (R + rows - 1) / rows * cols < 4 * g_num_sms) rows /= 2;
	const dim3 grid((R + rows - 1) / rows, cols);
	PT *o = static_cast<PT *>(out), *p = static_cast<PT *>(plain);
	if (taps <= 2) launch_k(norm_conv_kernel<PT, 2>, grid, dim3(128), 0, st, o, p, ldo, x, ldx, stats, w, cw, hist, d, R, D, taps, rows);
	else if (taps <= 4) launch_k(norm_conv_kernel<PT, 4>, grid, dim3(128), 0, st, o, p, ldo, x, ldx, stats, w, cw, hist, d, R, D, taps, rows);
	else launch_k(norm_conv_kernel<PT, 16>, grid, dim3(128), 0, st, o, p, ldo, x, ldx, stats, w, cw, hist, d, R, D, taps, rows);
	count_launch();
	return check_launch("norm_conv");
}
template <typename PT> int launch_norm(void *out, int ldo, const float *x, int ldx, const float *w, const int *rows, int n, int D, float eps, int rms, float *out32,
                                       cudaStream_t st) {
	launch_k(row_norm_kernel<PT>, dim3(n), dim3(128), 0, st, static_cast<PT *>(out), ldo, x, ldx, w, rows, n, D, eps, rms, out32);
	count_launch();
	return check_launch("row_norm");
}
// n_exp: CTAs per row of its chosen experts (0: the step's experts are grouped products)
template <typename PT, typename CT, typename OT> int launch_beside_mix(const WAttnArgs *w, const LinArgs *l, const MoeArgs &e, int n_exp, int R, cudaStream_t st) {
	const size_t ex = n_exp ? expert_token_smem(e.D) : 0;
	const int n_mix = w ? w->G * w->nsplit : lin_token_ctas(l->H, l->vd);
	const size_t smem = std::max(ex, w ? wattn_token_smem(w->H / w->G, w->dkp, w->dvp) : lin_token_smem(l->Np));
	const dim3 grid(n_mix + n_exp, R);
	const WAttnArgs wa = w ? *w : WAttnArgs{};
	const LinArgs la = l ? *l : LinArgs{};
	auto go = [&](auto kernel) -> int {
		TG_TRY(allow_smem(kernel, smem));
		launch_k(kernel, grid, dim3(256), smem, st, wa, la, e, n_mix);
		return TG_OK;
	};
	if (w) TG_TRY(n_exp ? go(beside_token_mix_kernel<PT, CT, OT, true, true>) : go(beside_token_mix_kernel<PT, CT, OT, true, false>));
	else TG_TRY(n_exp ? go(beside_token_mix_kernel<PT, CT, OT, false, true>) : go(beside_token_mix_kernel<PT, CT, OT, false, false>));
	count_launch();
	return check_launch("beside_token_mix");
}
// portions of a recurrence: its inputs
template <typename PT, int V> int launch_lin_conv(const LinArgs &a, int R, cudaStream_t st) {
	const int cols = (a.ldxc + 128 * V - 1) / (128 * V) + 1;
	int rows = LV_ROWS;
	while (rows > 1 && (R + rows - 1) / rows * cols < 4 * g_num_sms) rows /= 2;
	const dim3 grid((R + rows - 1) / rows, cols);
	if (a.taps <= 4) launch_k(lin_conv_kernel<PT, 4, V>, grid, dim3(128), 0, st, a, R, rows);
	else launch_k(lin_conv_kernel<PT, 16, V>, grid, dim3(128), 0, st, a, R, rows);
	count_launch();
	return check_launch("lin_conv");
}
template <typename PT> int launch_lin_inputs(const LinArgs &a, int R, int nseg, cudaStream_t st) {
	if (a.kind == LIN_SSM) return a.vd % 4 == 0 && a.N % 4 == 0 && a.p_x % 4 == 0 ? launch_lin_conv<PT, 4>(a, R, st) : launch_lin_conv<PT, 1>(a, R, st);
	launch_k(lin_gates_kernel, dim3(a.H, nseg), dim3(LG_THREADS), 0, st, a);
	count_launch();
	return check_launch("lin_gates");
}
template <typename PT> int launch_lin_scan(const LinArgs &a, int nseg, cudaStream_t st) {
	const dim3 grid((a.vd + LT_COLS - 1) / LT_COLS, a.H, nseg);
	if (a.N <= 128) launch_k(lin_scan_kernel<PT, 4>, grid, dim3(256), 0, st, a);
	else if (a.N <= 256) launch_k(lin_scan_kernel<PT, 8>, grid, dim3(256), 0, st, a);
	else launch_k(lin_scan_kernel<PT, 16>, grid, dim3(256), 0, st, a);
	count_launch();
	return check_launch("lin_scan");
}
int launch_lin_chunks(LinArgs a, const CUtensorMap &rows, const CUtensorMap &sh, const CUtensorMap &sl, int nseg, int max_len, cudaStream_t st) {
	const int chunks = (max_len + LC - 1) / LC, tiles = (a.vdp + 63) / 64;
	TG_TRY(allow_smem(lin_chunk_state_kernel, lin_state_smem(a.Np)));
	launch_k(lin_chunk_state_kernel, dim3(chunks, a.H * tiles, nseg), dim3(256), lin_state_smem(a.Np), st, rows, a);
	count_launch();
	TG_TRY(check_launch("lin_chunk_state"));
	const int items = a.H * a.N * (a.vdp / 4) + (a.kind == LIN_MLSTM ? a.H * a.N : 0);
	launch_k(lin_chunk_scan_kernel, dim3((items + 255) / 256, nseg), dim3(256), 0, st, a);
	count_launch();
	TG_TRY(check_launch("lin_chunk_scan"));
	// (few chunks: more CTAs share a head's columns, each forming the weights again)
	a.vsplit = std::max(1, std::min(tiles, g_num_sms / std::max(1, chunks * a.H * nseg)));
	TG_TRY(allow_smem(lin_chunk_out_kernel, lin_out_smem(a.Np)));
	launch_k(lin_chunk_out_kernel, dim3(chunks, a.H * a.vsplit, nseg), dim3(256), lin_out_smem(a.Np), st, rows, sh, sl, a);
	count_launch();
	return check_launch("lin_chunk_out");
}
template <typename T> int launch_lin_norm(const LinArgs &a, const Layer &L, void *O, const void *P, int R, float eps, cudaStream_t st) {
	const int n = a.H * a.vd;
	auto go = [&](auto kernel) {
		launch_k(kernel, dim3((R * L.li.parts + 7) / 8), dim3(256), 0, st, static_cast<T *>(O), L.kcat, a.o, a.ldo, static_cast<const T *>(P) + L.p_z, L.ldp, L.rnorm, R, n,
		         L.li.parts, a.kind == LIN_SSM ? 1 : 0, eps);
	};
	if (n / L.li.parts % 4 == 0 && L.p_z % 4 == 0) go(lin_norm_kernel<T, 4>);
	else go(lin_norm_kernel<T, 1>);
	count_launch();
	return check_launch("lin_norm");
}
template <typename T> int launch_gather(const MoeArgs &a, const void *h, int ldh, void *xg, int R, cudaStream_t st) {
	const int rows = R >= 4 * MG_ROWS * g_num_sms ? MG_ROWS : 1;
	launch_k(expert_gather_kernel<T>, dim3((R + rows - 1) / rows), dim3(128), 0, st, a, static_cast<const T *>(h), ldh, static_cast<T *>(xg), R, rows);
	count_launch();
	return check_launch("expert_gather");
}
// portions on CUDA cores
template <typename PT> int launch_attn_simt(const WAttnArgs &a, int R, cudaStream_t st) {
	const size_t smem = size_t(4) * (a.dkp + a.dvp) * 4;
	TG_TRY(allow_smem(window_attn_kernel<PT, PT>, smem));
	launch_k(window_attn_kernel<PT, PT>, dim3((R * a.H + 3) / 4), dim3(128), smem, st, a, R);
	count_launch();
	return check_launch("window_attn");
}
}  // namespace

// attention of a portion, its keys and values being in the cache
int HybridState::attn_rows(const WAttnArgs &wa, int run, int R, int nseg, int max_len) {
	const int li = m->runs[run].layer;
	const RunCache &c = cache[run];
	static const int use_tc = env_int("TG_WATTN_TC", 1);
	if (!f32 && use_tc && wa.dkp <= 256 && wa.dvp <= 256) {
		const WtShape sh = wt_shape(wa.dkp, wa.dvp, wa.window, wa.r1 != nullptr);
		TG_TRY(allow_smem(window_attn_tc_kernel, sh.total));
		launch_k(window_attn_tc_kernel, dim3((max_len + 127) / 128, wa.H, nseg), dim3(WT_THREADS), size_t(sh.total), stream, pmap[li], c.kmap, c.vmap,
		         c.ksmap, c.vsmap, wa);
		count_launch();
		TG_TRY(check_launch("window_attn_tc"));
	} else {
		if (f32) TG_TRY(launch_attn_simt<float>(wa, R, stream));
		else TG_TRY(launch_attn_simt<bf16>(wa, R, stream));
	}
	return TG_OK;
}

// how many CTAs share the keys of a (sequence, key/value head) in a step of one token per sequence
int HybridState::token_splits(const WAttnArgs &wa, int fill) const {
	const long long second = wa.pool ? max_pos_global / wa.pool : wa.keep, keys = std::min<long long>(wa.window + second, max_pos_global);
	return int(std::max<long long>(1, std::min<long long>(std::min(nsplit_cap, fill), (keys + WK_KEYS - 1) / WK_KEYS)));
}

// rows up to which a step of one token per sequence is made of matrix-vector products
int HybridState::few_rows() const {
	static const int most = env_int("TG_FEW_ROWS", FEW_ROWS);
	return std::min(most, FEW_ROWS);
}

// ---- feed-forward after the mixer
int HybridState::few_layer(const StepDesc &d, int run, int R) {
	const Layer &L = m->layers[m->runs[run].layer];
	const RunCache &c = cache[run];
	const int D = m->D;
	GemvArgs g{};
	g.d = d;
	g.x = x;
	g.ldx = ldx;
	g.D = D;
	g.embed = m->embed.W;
	g.lde = m->embed.ld;
	g.V = m->n_vocab;
	g.eps = m->eps;
	g.cw = L.canon;
	g.hist = c.canon;
	g.taps = m->taps;
	g.act = L.ff.act;
	g.limit = L.ff.limit;
	const int embed_mode = run == 0 ? 1 : (m->runs[run].add_embed ? 2 : 0);
	auto product = [&](int pro, int epi, const Lin &w, const float *norm, const float *vec, int ldv, float *out, int ldo, int em) -> int {
		GemvArgs s = g;
		s.W = w.W;
		s.ldw = w.ld;
		s.N = w.N;
		s.K = w.K;
		s.w = norm;
		s.vec = vec;
		s.ldv = ldv;
		s.out = out;
		s.ldo = ldo;
		s.embed_mode = em;
		if (epi == GV_PROJ) {
			s.p_k = L.p_k;
			s.n_k = L.at.G * L.at.dkp;
			s.p_v = L.p_v;
			s.n_v = L.at.G * L.at.dvp;
			s.kc = c.kc;
			s.vc = c.vc;
			s.ks = c.ks;
			s.vs = c.vs;
			s.cap_rows = c.cap;
			s.keep = std::min(L.at.keep, c.keep_rows);
			s.keep_rows = c.keep_rows;
			s.cache_f32 = f32;
		}
		return gemv(pro, epi, s, R);
	};
	TG_TRY(product(GV_LN_CONV, GV_PROJ, L.proj, L.norm1, nullptr, 0, P32, L.ldp, embed_mode));
	WAttnArgs wa = attn_args(d, run, P32, L.ldp, O32, L.kc);
	const DeltaArgs da = delta_args(d, run, P32, L.ldp, O32, L.kc);
	wa.nsplit = token_splits(wa, nsplit_cap);
	if (f32) TG_TRY((launch_token_mix<float, float, float>(wa, da, R, stream)));
	else TG_TRY((launch_token_mix<float, bf16, float>(wa, da, R, stream)));
	TG_TRY(product(GV_VEC, GV_ADD, L.out, nullptr, O32, L.kc, x, ldx, embed_mode));
	if (L.ff.ff) {
		TG_TRY(product(GV_LN, GV_GLU, L.gu, L.norm2, nullptr, 0, act32, L.ff.ffp, 0));
		TG_TRY(product(GV_VEC, GV_ADD, L.down, nullptr, act32, L.ff.ffp, x, ldx, 0));
	}
	return TG_OK;
}

int HybridState::rows_layer(const StepDesc &d, int run, int R, int nseg, int max_len) {
	const int li = m->runs[run].layer, D = m->D;
	const Layer &L = m->layers[li];
	const bool single = max_len == 1;
	TG_TRY(norm_in(d, run, R));
	TG_TRY(gemm(GEMM_STORE, h, m->Dp, &hmap, L.proj, R, P, L.ldp));
	WAttnArgs wa = attn_args(d, run, P, L.ldp, O, L.kc);
	const DeltaArgs da = delta_args(d, run, P, L.ldp, O, L.kc);
	if (f32) launch_k(kv_append_kernel<float, float>, dim3(R), dim3(256), 0, stream, wa);
	else launch_k(kv_append_kernel<bf16, bf16>, dim3(R), dim3(256), 0, stream, wa);
	count_launch();
	TG_TRY(check_launch("kv_append"));
	if (single) {
		wa.nsplit = token_splits(wa, std::max(1, 2 * g_num_sms / std::max(1, R * wa.G)));
		if (f32) TG_TRY((launch_token_mix<float, float, float>(wa, da, R, stream)));
		else TG_TRY((launch_token_mix<bf16, bf16, bf16>(wa, da, R, stream)));
	} else {
		TG_TRY(attn_rows(wa, run, R, nseg, max_len));
		const size_t esz = f32 ? 4 : 2;
		const uint8_t *pb = static_cast<const uint8_t *>(P);
		TG_TRY(gemm(GEMM_STORE32, pb + size_t(L.p_a1) * esz, L.ldp, f32 ? nullptr : &a1map[li], L.a2, R, z, da.ldz));
		TG_TRY(gemm(GEMM_STORE32, pb + size_t(L.p_g1) * esz, L.ldp, f32 ? nullptr : &g1map[li], L.g2, R, gz, da.ldgz));
		if (f32) TG_TRY(launch_delta<float>(da, R, nseg, max_len, stream));
		else TG_TRY(launch_delta<bf16>(da, R, nseg, max_len, stream));
	}
	TG_TRY(gemm(GEMM_ADD, O, L.kc, f32 ? nullptr : &omap[li], L.out, R, x, ldx));
	if (L.ff.ff) {
		if (f32) TG_TRY(launch_norm<float>(h, m->Dp, x, ldx, L.norm2, nullptr, R, D, m->eps, m->rms, nullptr, stream));
		else TG_TRY(launch_norm<bf16>(h, m->Dp, x, ldx, L.norm2, nullptr, R, D, m->eps, m->rms, nullptr, stream));
		GemmOpt glu_opt;
		glu_opt.act = L.ff.act;
		glu_opt.limit = L.ff.limit;
		TG_TRY(gemm(GEMM_GLU, h, m->Dp, &hmap, L.gu, R, act, L.ff.ffp, glu_opt));
		TG_TRY(gemm(GEMM_ADD, act, L.ff.ffp, f32 ? nullptr : &amap[li], L.down, R, x, ldx));
	}
	return TG_OK;
}

// ---- feed-forward beside the mixer
int HybridState::beside_few_layer(const StepDesc &d, int run, int R) {
	const Layer &L = m->layers[m->runs[run].layer];
	const RunCache &c = cache[run];
	const FfSpec &F = L.ff;
	const bool lin_mix = L.li.H > 0;
	GemvArgs g{};
	g.d = d;
	g.x = x;
	g.ldx = ldx;
	g.D = m->D;
	g.embed = m->embed.W;
	g.lde = m->embed.ld;
	g.V = m->n_vocab;
	g.eps = m->eps;
	g.embed_mode = run == 0 ? 1 : 0;
	g.act = F.act;
	g.limit = F.limit;
	GemvArgs f = g;
	f.W = L.front.W;
	f.ldw = L.front.ld;
	f.N = L.front.N;
	f.K = L.front.K;
	f.w = L.norm1;
	f.cw = L.canon;
	f.hist = c.canon;
	f.taps = m->taps;
	f.out = P32;
	f.ldo = L.ldp;
	f.n_proj = L.proj.N;
	f.n32 = L.n32;
	f.out32 = T32;
	f.ld32 = L.tail();
	f.n_glu = F.ffp;
	f.glu_out = O32 + L.kc;
	f.ld_glu = L.kcat;
	f.n_route = F.experts;
	f.route_out = RL;
	f.ld_route = round_up(F.experts, 8);
	f.norm_out = F.experts ? h32 : nullptr;
	TG_TRY(gemv(GV_LN_CONV, GV_FRONT, f, R));
	const MoeArgs ma = moe_args(L);
	const int n_exp = F.experts ? expert_token_ctas(F.top, F.effp) : 0;
	if (lin_mix) {
		LinArgs la = lin_args(d, run, P32);
		la.o = O32;
		la.ldo = L.kcat;
		TG_TRY((launch_beside_mix<float, float, float>(nullptr, &la, ma, n_exp, R, stream)));
	} else {
		WAttnArgs wa = attn_args(d, run, P32, L.ldp, O32, L.kcat);
		wa.append = 1;
		wa.nsplit = token_splits(wa, nsplit_cap);
		if (f32) TG_TRY((launch_beside_mix<float, float, float>(&wa, nullptr, ma, n_exp, R, stream)));
		else TG_TRY((launch_beside_mix<float, bf16, float>(&wa, nullptr, ma, n_exp, R, stream)));
	}
	GemvArgs o = g;
	o.W = L.out.W;
	o.ldw = L.out.ld;
	o.N = L.out.N;
	o.K = L.out.K;
	o.vec = O32;
	o.ldv = L.kcat;
	o.out = x;
	o.ldo = ldx;
	o.w = L.rnorm;
	if (lin_mix) {
		o.mix_norm = L.li.kind == LIN_SSM ? MIX_GATE_NORM : MIX_NORM_GATE;
		o.mix_n = L.li.H * L.li.vd;
		o.parts = L.li.parts;
		o.gate = P32 + L.p_z;
		o.ldg = L.ldp;
	}
	if (F.experts) {
		o.top = F.top;
		o.n_ex = F.effp;
		o.ex_act = ex32;
		o.ex_w = moe.w;
		o.ex_id = moe.id;
		o.ex_W = L.ex_down.W;
		o.ld_ex = L.ex_down.ld;
	}
	return gemv(GV_MIX, GV_ADD, o, R);
}

int HybridState::beside_rows_layer(const StepDesc &d, int run, int R, int nseg, int max_len) {
	const int li = m->runs[run].layer;
	const Layer &L = m->layers[li];
	const FfSpec &F = L.ff;
	const bool single = max_len == 1;
	TG_TRY(norm_in(d, run, R));
	GemmOpt po;
	po.n32 = L.n32;
	po.ld32 = L.tail();
	po.C32 = L.tail() ? T32 : nullptr;
	TG_TRY(gemm(GEMM_STORE, h, m->Dp, &hmap, L.proj, R, P, L.ldp, po));
	if (L.at.H) {
		WAttnArgs wa = attn_args(d, run, P, L.ldp, O, L.kcat);
		if (single) {
			wa.append = 1;
			wa.nsplit = token_splits(wa, std::max(1, 2 * g_num_sms / std::max(1, R * wa.G)));
			if (f32) TG_TRY((launch_beside_mix<float, float, float>(&wa, nullptr, MoeArgs{}, 0, R, stream)));
			else TG_TRY((launch_beside_mix<bf16, bf16, bf16>(&wa, nullptr, MoeArgs{}, 0, R, stream)));
		} else {
			const int unit = wa.pool ? wa.pool * std::max(1, 16 / wa.pool) : 16;
			const dim3 grid((max_len + unit - 1) / unit + 1, wa.G, nseg);
			if (f32) launch_k(kv_transform_kernel<float, float>, grid, dim3(256), 0, stream, wa, unit);
			else launch_k(kv_transform_kernel<bf16, bf16>, grid, dim3(256), 0, stream, wa, unit);
			count_launch();
			TG_TRY(check_launch("kv_transform"));
			TG_TRY(attn_rows(wa, run, R, nseg, max_len));
		}
	} else {
		LinArgs la = lin_args(d, run, P);
		if (single) {
			if (la.kind == LIN_SSM) {
				la.ready = 1;
				TG_TRY(f32 ? launch_lin_inputs<float>(la, R, nseg, stream) : launch_lin_inputs<bf16>(la, R, nseg, stream));
			}
			if (f32) TG_TRY((launch_beside_mix<float, float, float>(nullptr, &la, MoeArgs{}, 0, R, stream)));
			else TG_TRY((launch_beside_mix<bf16, bf16, bf16>(nullptr, &la, MoeArgs{}, 0, R, stream)));
		} else {
			if (f32) TG_TRY(launch_lin_inputs<float>(la, R, nseg, stream));
			else TG_TRY(launch_lin_inputs<bf16>(la, R, nseg, stream));
			if (lin_tc && la.Np <= 256 && max_len > LIN_SCAN_MAX)
				TG_TRY(launch_lin_chunks(la, la.kind == LIN_SSM ? xcmap[li] : pmap[li], shmap[li], slmap[li], nseg, max_len, stream));
			else if (f32) TG_TRY(launch_lin_scan<float>(la, nseg, stream));
			else TG_TRY(launch_lin_scan<bf16>(la, nseg, stream));
		}
		if (f32) TG_TRY(launch_lin_norm<float>(la, L, O, P, R, m->eps, stream));
		else TG_TRY(launch_lin_norm<bf16>(la, L, O, P, R, m->eps, stream));
	}
	if (F.any()) {
		GemmOpt go;
		go.act = F.act;
		go.limit = F.limit;
		go.n32 = 2 * F.ffp;
		go.C32 = F.experts ? RL : nullptr;
		go.ld32 = round_up(F.experts, 8);
		uint8_t *dst = static_cast<uint8_t *>(O) + size_t(L.kc) * (f32 ? 4 : 2);
		TG_TRY(gemm(GEMM_GLU, hp, m->Dp, &hpmap, L.gu, R, dst, L.kcat, go));
	}
	if (F.experts) {
		const MoeArgs ma = moe_args(L);
		const int rounds = std::max(1, std::min(MR_ROUNDS, R / (8 * g_num_sms)));
		launch_k(route_kernel, dim3((R + 8 * rounds - 1) / (8 * rounds)), dim3(256), 0, stream, ma, R, rounds);
		count_launch();
		TG_TRY(check_launch("route"));
		if (f32) TG_TRY(launch_gather<float>(ma, hp, m->Dp, xg, R, stream));
		else TG_TRY(launch_gather<bf16>(ma, hp, m->Dp, xg, R, stream));
		GemmOpt eo;
		eo.act = F.act;
		eo.limit = F.limit;
		eo.grouped = true;
		const int most = moe_rows(L, R);
		eo.est = std::max(1, R * F.top / GB_BM + std::min(F.experts, R * F.top) / 2);
		TG_TRY(gemm(GEMM_GLU, xg, m->Dp, &xgmap, L.ex_gu, most, xa, F.effp, eo));
		TG_TRY(gemm(GEMM_STORE, xa, F.effp, f32 ? nullptr : &xamap[li], L.ex_down, most, xy, ldx, eo));
	}
	int bn = 0, splits = 1;
	if (!f32) pick_split(R, m->D, L.kcat, &bn, &splits);
	left.experts = F.experts ? li : -1;
	if (splits > 1 && size_t(splits) * R <= split_rows) {
		GemmOpt so;
		so.splits = left.parts = splits;
		so.bn = bn;
		return gemm(GEMM_STORE32, O, L.kcat, &omap[li], L.out, R, split_part, ldx, so);
	}
	return gemm(GEMM_ADD, O, L.kcat, f32 ? nullptr : &omap[li], L.out, R, x, ldx);
}

template <typename T> RowSum<T> HybridState::row_sum(int R) {
	RowSum<T> add{};
	if (left.experts >= 0) {
		add.y = static_cast<const T *>(xy);
		add.ldy = ldx;
		add.top = m->layers[left.experts].ff.top;
		add.slot = moe.place;
		add.w = moe.w;
	}
	add.part = split_part;
	add.n_part = left.parts;
	add.part_stride = size_t(R) * ldx;
	left = Left();
	return add;
}

int HybridState::norm_in(const StepDesc &d, int run, int R) {
	const Layer &L = m->layers[m->runs[run].layer];
	float *hist = cache[run].canon;
	void *plain = L.beside ? hp : nullptr;
	auto go = [&](auto t) -> int {
		typedef decltype(t) T;
		RowSum<T> add = row_sum<T>(R);
		if (L.ff.experts) {
			add.zero = moe.count;
			add.n_zero = L.ff.experts;
		}
		TG_TRY(launch_stats<T>(stats, x, ldx, R, m->D, m->eps, m->rms, add, stream));
		return launch_norm_conv<T>(h, plain, m->Dp, x, ldx, stats, L.norm1, L.canon, hist, d, R, m->D, m->taps, stream);
	};
	return f32 ? go(0.0f) : go(bf16());
}

// adds to the stream what is left to be added (where no norm follows that would do it)
int HybridState::add_left(int R) {
	if (left.experts < 0 && !left.parts) return TG_OK;
	if (f32) return launch_stats<float>(stats, x, ldx, R, m->D, m->eps, m->rms, row_sum<float>(R), stream);
	return launch_stats<bf16>(stats, x, ldx, R, m->D, m->eps, m->rms, row_sum<bf16>(R), stream);
}

// All layers for R rows in nseg segments (the longest: max_len), leaving the residual stream in x.
int HybridState::run_layers(const StepDesc &d, int R, int nseg, int max_len) {
	const bool few = max_len == 1 && R <= few_rows();
	const int D = m->D;
	auto embed_rows = [&](int add) -> int {
		launch_k(embed_rows_kernel, dim3(R), dim3(256), 0, stream, x, ldx, m->embed.W, m->embed.ld, m->embed_scale, d, D, m->n_vocab, add, err_flag);
		count_launch();
		return check_launch("embed_rows");
	};
	if (!few) TG_TRY(embed_rows(0));
	if (!m->rots.empty()) {
		RopeTable t{m->rot_freq, m->rot_factor, cs, max_rows, m->rot_half};
		launch_k(rope_table_kernel, dim3(R, int(m->rots.size())), dim3(128), 0, stream, t, d);
		count_launch();
		TG_TRY(check_launch("rope_table"));
	}
	left = Left();
	for (size_t run = 0; run < m->runs.size(); run++) {
		const Layer &L = m->layers[m->runs[run].layer];
		if (few) {
			TG_TRY(L.beside ? beside_few_layer(d, int(run), R) : few_layer(d, int(run), R));
		} else {
			if (m->runs[run].add_embed) TG_TRY(embed_rows(1));
			if (L.beside) TG_TRY(beside_rows_layer(d, int(run), R, nseg, max_len));
			else TG_TRY(rows_layer(d, int(run), R, nseg, max_len));
			if (tracing || run + 1 == m->runs.size()) TG_TRY(add_left(R));
		}
		if (tracing) {
			const size_t at = trace.size();
			trace.resize(at + size_t(R) * D);
			TG_CUDA(cudaMemcpy2DAsync(trace.data() + at, size_t(D) * 4, x, size_t(ldx) * 4, size_t(D) * 4, R, cudaMemcpyDeviceToHost, stream));
			TG_CUDA(cudaStreamSynchronize(stream));
		}
	}
	return TG_OK;
}

// logits of n rows of x (rows_dev: which; null: 0 .. n-1) -> out [n][ld_logits]
int HybridState::score_rows(const int *rows_dev, int n, float *out, float *norm_out) {
	if (f32) TG_TRY(launch_norm<float>(hn, m->Dp, x, ldx, m->final_norm, rows_dev, n, m->D, m->eps, m->rms, norm_out, stream));
	else TG_TRY(launch_norm<bf16>(hn, m->Dp, x, ldx, m->final_norm, rows_dev, n, m->D, m->eps, m->rms, norm_out, stream));
	GemmOpt o;
	o.cap = m->softcap;
	return gemm(GEMM_LOGITS, hn, m->Dp, &hnmap, m->head, n, out, ld_logits, o);
}

// ------------------------------------------------------------------ lock-step decoding
int HybridState::enqueue_decode_all() {
	const StepDesc d = lockstep_desc();
	TG_TRY(run_layers(d, B, B, 1));
	if (B <= few_rows()) {
		GemvArgs g{};
		g.d = d;
		g.x = x;
		g.ldx = ldx;
		g.D = m->D;
		g.W = m->head.W;
		g.ldw = m->head.ld;
		g.N = m->head.N;
		g.K = m->head.K;
		g.w = m->final_norm;
		g.eps = m->eps;
		g.taps = 1;
		g.out = logits;
		g.ldo = ld_logits;
		g.norm_out = xnorm;
		g.cap = m->softcap;
		TG_TRY(gemv(GV_LN, GV_LOGITS, g, B));
	} else {
		TG_TRY(score_rows(nullptr, B, logits, xnorm));
	}
	launch_k(hybrid_advance_kernel, dim3((B + 255) / 256), dim3(256), 0, stream, ls_pos, ls_par, B);
	count_launch();
	return check_launch("hybrid_advance");
}

int HybridState::enqueue_forward() {
	TG_TRY(sync_lockstep());
	if (tracing) {
		trace.clear();
		trace_rows = B;
		TG_TRY(enqueue_decode_all());
	} else {
		TG_TRY(enqueue_decode_step());
	}
	for (int &p : host_par) p ^= 1;
	return TG_OK;
}

int HybridState::run_steps(int n_steps, float minp, float temp) {
	TG_TRY(sync_lockstep());
	TG_TRY(tg_state::run_steps(n_steps, minp, temp));
	if (n_steps & 1)
		for (int &p : host_par) p ^= 1;
	return TG_OK;
}

// ------------------------------------------------------------------ portions
int HybridState::run_entries(std::vector<Entry> &es, bool last, float *logits_host) {
	TG_CUDA(cudaStreamSynchronize(stream));
	staging_busy = false;
	trace.clear();
	trace_rows = 0;
	ls_dirty = true;
	for (;;) {
		// a pass: what fits of every entry that has tokens left
		int R = 0, nseg = 0, max_len = 0;
		int *tk = desc_pin, *rs = tk + max_rows, *sg = rs + max_rows;
		struct Out {
			size_t entry;
			int row;
			size_t out;
		};
		std::vector<Out> outs;
		for (size_t e = 0; e < es.size(); e++) {
			Entry &E = es[e];
			const int n = std::min(std::min(E.count - E.done, max_seq_rows), max_rows - R);
			if (n <= 0) continue;
			for (int i = 0; i < n; i++) {
				tk[R + i] = E.ids[E.done + i];
				rs[R + i] = nseg;
			}
			sg[nseg] = E.seq;
			sg[B + nseg] = R;
			sg[2 * B + nseg] = n;
			sg[3 * B + nseg] = host_pos[E.seq];
			sg[4 * B + nseg] = host_par[E.seq];
			if (last) {
				if (E.done + n == E.count) outs.push_back({e, R + n - 1, size_t(E.seq)});
			} else {
				for (size_t w = 0; w < E.want.size(); w++)
					if (E.want[w] >= E.done && E.want[w] < E.done + n) outs.push_back({e, R + E.want[w] - E.done, E.out0 + w});
			}
			host_pos[E.seq] += n;
			host_par[E.seq] ^= 1;
			E.done += n;
			R += n;
			nseg++;
			max_len = std::max(max_len, n);
		}
		if (R == 0) break;
		TG_CUDA(cudaMemcpyAsync(desc, desc_pin, desc_ints * 4, cudaMemcpyHostToDevice, stream));
		StepDesc d;
		d.tok = desc;
		d.row_seg = desc + max_rows;
		d.seg_seq = desc + 2 * size_t(max_rows);
		d.seg_row = d.seg_seq + B;
		d.seg_len = d.seg_seq + 2 * B;
		d.seg_pos = d.seg_seq + 3 * B;
		d.seg_par = d.seg_seq + 4 * B;
		trace_rows += R;
		TG_TRY(run_layers(d, R, nseg, max_len));
		for (size_t i = 0; i < outs.size();) {
			// a run of consecutive output rows
			std::vector<int> rows{outs[i].row};
			while (i + rows.size() < outs.size() && rows.size() < size_t(wl_rows) && outs[i + rows.size()].out == outs[i].out + rows.size())
				rows.push_back(outs[i + rows.size()].row);
			const int n = int(rows.size());
			TG_CUDA(cudaMemcpyAsync(want_dev, rows.data(), size_t(n) * 4, cudaMemcpyHostToDevice, stream));
			if (last) {
				TG_TRY(score_rows(want_dev, n, logits + outs[i].out * ld_logits, xnorm + outs[i].out * m->D));
			} else {
				TG_TRY(score_rows(want_dev, n, wl, nullptr));
				const size_t row = size_t(m->n_vocab) * 4;
				TG_CUDA(cudaMemcpy2DAsync(logits_host + outs[i].out * m->n_vocab, row, wl, size_t(ld_logits) * 4, row, n, cudaMemcpyDeviceToHost, stream));
			}
			i += size_t(n);
		}
		TG_TRY(check_err_flag());  // synchronises: the pinned descriptors may be rewritten
	}
	if (last && logits_host) {
		TG_TRY(read_logits(logits_host));
		TG_CUDA(cudaStreamSynchronize(stream));
	}
	return TG_OK;
}

int HybridState::prefill(const int *ids, int S, float *logits_host) {
	for (long long i = 0; i < (long long)B * S; i++)
		if (ids[i] < 0 || ids[i] >= m->n_vocab) return fail(TG_EINVAL, "token id out of range");
	std::vector<Entry> es(B);
	for (int b = 0; b < B; b++) {
		es[b].seq = b;
		es[b].count = S;
		es[b].done = 0;
		es[b].ids = ids + size_t(b) * S;
		es[b].out0 = 0;
	}
	return run_entries(es, true, logits_host);
}

int HybridState::append(const int *ids, int n, float *logits_host) {
	std::vector<Entry> es(1);
	es[0].seq = 0;
	es[0].count = n;
	es[0].done = 0;
	es[0].ids = ids;
	es[0].out0 = 0;
	return run_entries(es, true, logits_host);
}

int HybridState::step(int n, const int *seq, const int *count, const int *ids, const int *n_want, const int *want, float *logits_host) {
	std::vector<Entry> es(n);
	std::vector<char> used(B, 0);
	size_t at = 0, out = 0;
	bool in_order = n == B;
	for (int e = 0; e < n; e++) {
		Entry &E = es[e];
		if (seq[e] < 0 || seq[e] >= B || used[seq[e]]) return fail(TG_EINVAL, "tg_step: bad or repeated sequence");
		if (count[e] < 1) return fail(TG_EINVAL, "tg_step: an entry without tokens");
		used[seq[e]] = 1;
		if (count[e] > max_pos_global - host_pos[seq[e]]) return fail(TG_ESTATE, "cache full (max_pos_global reached)");
		E.seq = seq[e];
		E.count = count[e];
		E.done = 0;
		E.ids = ids + at;
		for (int i = 0; i < count[e]; i++)
			if (E.ids[i] < 0 || E.ids[i] >= m->n_vocab) return fail(TG_EINVAL, "token id out of range");
		E.out0 = out;
		for (int w = 0; n_want && w < n_want[e]; w++) {
			const int p = want[out + w];
			if (p < 0 || p >= count[e]) return fail(TG_EINVAL, "tg_step: a wanted place outside the entry");
			E.want.push_back(p);
		}
		at += count[e];
		out += E.want.size();
		in_order = in_order && seq[e] == e && count[e] == 1;
	}
	if (out && !logits_host) return fail(TG_EINVAL, "tg_step: no buffer for the logits");
	if (!in_order) return run_entries(es, false, logits_host);
	// one token for every sequence: the decode step of the generation loop
	TG_TRY(staging_acquire());
	std::memcpy(host_pin, ids, 4 * size_t(B));
	TG_CUDA(cudaMemcpyAsync(tok, host_pin, 4 * size_t(B), cudaMemcpyHostToDevice, stream));
	TG_TRY(enqueue_forward());
	for (int b = 0; b < B; b++) {
		host_pos[b] += 1;
		for (size_t w = 0; w < es[b].want.size(); w++)
			TG_CUDA(cudaMemcpyAsync(logits_host + (es[b].out0 + w) * m->n_vocab, logits + size_t(b) * ld_logits, size_t(m->n_vocab) * 4, cudaMemcpyDeviceToHost, stream));
	}
	return check_err_flag();
}
