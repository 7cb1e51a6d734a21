// What the model families of libtinygemma_b200 share on the host side: error handling, launch helpers, and the
// two base classes behind the C ABI's handles. tg_core.cu implements the family-independent entry points (state
// life cycle, samplers, generation loops, the architecture registry) in terms of the virtual functions below;
// tg_gemma.cu and tg_hybrid.cu implement the families.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

#include "../../include/tiny_gemma_b200.h"

namespace tg {

// ------------------------------------------------------------------ errors, counters, environment (tg_core.cu)
int fail(int code, const std::string &msg);
void count_launch(int n = 1);
long long launches();           // kernels launched so far
void set_launches(long long n); // (a captured graph's launches count at replay, not at capture)
int check_launch(const char *what);
int env_int(const char *name, int dflt);  // tunables for experiments; defaults are the tuned values
int ensure_device(int device);
extern int g_num_sms;

#define TG_CUDA(call)                                                                                        \
	do {                                                                                                     \
		cudaError_t e__ = (call);                                                                            \
		if (e__ != cudaSuccess) return tg::fail(TG_ECUDA, std::string(#call) + ": " + cudaGetErrorString(e__)); \
	} while (0)

#define TG_TRY(call)                    \
	do {                                \
		int rc__ = (call);              \
		if (rc__ != TG_OK) return rc__; \
	} while (0)

// cudaFuncSetAttribute is per device: "configured once" flags are kept per device index
constexpr int TG_MAX_DEVICES = 64;
inline int current_device_slot() {
	int d = 0;
	cudaGetDevice(&d);
	return (d >= 0 && d < TG_MAX_DEVICES) ? d : 0;
}

// Launch with the programmatic-serialization attribute (see pdl_wait in tg_common.cuh): only for kernels that
// call pdl_wait() before their first global access. TG_PDL=0 launches them as ordinary stream-ordered kernels.
// Gemma's batched decode step switches it off for its own launches (g_pdl_scope_off): replayed from a CUDA graph
// that step gains nothing from it (measured 3.72 ms with ordinary edges, 3.78 ms with programmatic ones at 256
// sequences), while the eagerly launched prefill does (178 tokens: 4.00 -> 3.80 ms).
extern thread_local bool g_pdl_scope_off;
template <typename... KArgs, typename... Args>
inline void launch_k(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args &&...args) {
	static const int use_env = env_int("TG_PDL", 1);
	const int use = use_env && !g_pdl_scope_off;
	cudaLaunchConfig_t cfg = {};
	cfg.gridDim = grid;
	cfg.blockDim = block;
	cfg.dynamicSmemBytes = smem;
	cfg.stream = st;
	cudaLaunchAttribute at[1];
	at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
	at[0].val.programmaticStreamSerializationAllowed = 1;
	cfg.attrs = at;
	cfg.numAttrs = use ? 1 : 0;
	cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);  // errors surface in check_launch (cudaGetLastError)
}

typedef CUresult (*PFN_encodeTiled)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *,
                                    const cuuint64_t *, const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave,
                                    CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
PFN_encodeTiled get_encode_fn();

constexpr int STEP_RANDF = 64;  // uniforms per sequence that the per-step block of a state holds

struct SampleArgs;

}  // namespace tg

// ===================================================================== handles of the C ABI
struct tg_model {
	int device = 0;
	int n_vocab = 0;
	int hidden_size = 0;
	int n_pos = 0;  // most positions a state may hold
	virtual ~tg_model() {}
	virtual const char *arch() const = 0;
	virtual int new_state(int batch, int max_pos, tg_state **out) = 0;
};

// One batch of independent sequences: what sampling and the generation loops need, for every family.
struct tg_state {
	tg_model *model = nullptr;
	int B = 1;
	int max_pos_global = 0;            // positions a sequence may reach
	cudaStream_t stream = nullptr;
	float *logits = nullptr;           // [B][ld_logits]
	int ld_logits = 0;                 // n_vocab rounded up to a multiple of 4; the surplus entries are -inf
	float *xnorm = nullptr;            // [B][hidden] final-normed hidden state (read-back)
	int *tok = nullptr;                // [B] token of the next step
	int *tok_log = nullptr;            // [log_cap][B]
	int log_cap = 0;
	int *log_count = nullptr;          // [B]
	float *randf = nullptr;            // [randf_cap][B]
	int randf_cap = 0;
	int randf_valid = 0;               // uniforms per sequence uploaded so far (the largest upload)
	// One allocation holds the small per-step words, so that a step's inputs go up in ONE copy and its
	// results come back in ONE: [err_flag, 3 pad][tok B][randf_count B][log_count B][randf STEP_RANDF x B]
	int *step_blk = nullptr;
	bool randf_in_blk = false;         // randf still points into step_blk (it moves out when it has to grow)
	float *randf_blk = nullptr;        // the block's own STEP_RANDF x B uniforms
	bool lean_randf = false;           // the next one-token launch draws from randf_blk
	int *randf_count = nullptr;        // [B]
	int *err_flag = nullptr;
	int *host_pin = nullptr;           // pinned staging, 64 KiB
	bool staging_busy = false;         // an enqueued copy may still read host_pin (set by the asynchronous tg_decode)
	// decode graph
	cudaGraphExec_t graph = nullptr;
	bool use_graph = true;
	bool warmed = false;
	int graph_launches = 0;
	std::vector<int> host_pos;         // tokens each sequence holds

	virtual ~tg_state() {}
	int alloc_common();                // everything above (model, B and max_pos_global are set)
	void free_common();

	virtual int ready() { return TG_OK; }                       // may it compute yet?
	virtual int reset() = 0;                                    // the family's own counters; the caller synchronises
	virtual int prefill(const int *ids, int S, float *logits_host) = 0;
	virtual int append(const int *ids, int n, float *logits_host) = 0;
	virtual int enqueue_decode_all() = 0;                       // one token per sequence, fed from `tok`
	virtual int enqueue_forward() { return enqueue_decode_step(); }
	virtual int enqueue_sampler(float minp, float temp, bool log_tokens);
	virtual int run_steps(int n_steps, float minp, float temp);  // n_steps of forward + sampler, tokens logged
	virtual bool lean_step() const { return false; }            // run_steps(1) can draw its uniform from randf_blk
	virtual int report_err(int flag);                           // what the family's kernels left in err_flag
	virtual int step(int n, const int *seq, const int *count, const int *ids, const int *n_want, const int *want, float *logits_host);
	virtual int free_sequence(int b);
	virtual int trace_enable(int on);
	virtual int trace_read(float *x_host, size_t cap_floats, int *runs, int *tokens);

	int enqueue_decode_step();                                  // enqueue_decode_all, as a CUDA graph from the second call on
	int staging_acquire();
	int check_err_flag();
	int ensure_log(int steps);
	int read_logits(float *logits_host);                        // enqueue the copy [B][n_vocab]
	tg::SampleArgs sample_args(float minp, float temp, bool log_tokens);
};

namespace tg {
// ------------------------------------------------------------------ architecture registry
// A family registers how to open a model folder whose config.json names one of its architectures.
typedef int (*OpenFn)(const char *dir, int device, int dtype, tg_model **out);
struct RegisterArch {
	RegisterArch(const char *name, OpenFn fn);
};
}  // namespace tg
