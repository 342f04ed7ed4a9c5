// duletar.cu — the Duletar family of the model registry (family.h): a pre-norm decoder described by a config.json whose layers each
// carry ONE token mixer, chosen per layer, and an optional feed-forward:
//
//   mixer "latent_attention"    softmax attention whose keys and values are expanded per head from a low-rank latent c = rmsnorm(W_dkv h);
//                               queries pass a latent of their own; each head has d plain and r rotated query/key entries, the rotated
//                               key part is one vector shared by all heads; causal, no window
//   mixer "latent_attention_2"  the same without positions, with a sigmoid output gate; a layer may read another layer's latents
//                               ("kv_from") through expansions of its own
//   mixer "retention"           linear attention with one fixed decay per head: S_t = decay_h S_{t-1} + k_t v_t^T, o_t = S_t^T q_t, rotary
//                               positions on q and k, o over its root mean square, silu output gate
//   feed-forward                dense W_down relu(W_up h)^2, or a mixture of clamped gated experts: softmax scores over all experts, groups
//                               scored by their best expert limit the choice, weights = chosen scores over their sum
//
// x <- x + mixer(rmsnorm(x) w1), x <- x + ff(rmsnorm(x) w2); the embedding row is scaled; logits = cap * tanh(head . rmsnorm(x) / cap).
//
// The step function, graph replay of one-token steps, uploads, release and the C entry points are the shared sequence engine's
// (seq_family.cuh), the latent mixers' kernels in order are seq_latent.cuh's.  Per pass and layer here:
//     latent attention: norm -> rows product [dq | dkv | gate] -> latent_post (latent norms, rotated key, cache row) -> rows product [uq]
//                       -> batched per-head product with uk^T (queries into the latent) + rope_heads (rotated query part) -> swa_attn /
//                       swa_tile with ONE key/value head reading the cache rows in place -> batched per-head product with uv (gate fused)
//                       -> rows product [o] with the residual add fused
//     retention:        norm -> rows product [q | k | v | gate] -> rope_heads in place -> hgrn2 kernels in their fixed-decay mode (norm and
//                       gate fused) -> rows product [o] + residual
//     dense ff:         norm -> rows product [up, relu^2 fused] -> rows product [down] + residual
//     experts:          norm -> moe_router -> moe_sort -> moe_gemm [gate | up, clamped GLU fused] -> moe_gemm [down] -> moe_combine (+ residual)
//
// Cache / state manager: a latent-attention layer keeps ONE row of kv_rank + rot_dim elements per position (the normed latent and the
// rotated shared key), nothing per head; a layer with kv_from keeps nothing and reads the other layer's rows.  A retention layer keeps
// its fp32 state (heads x dim x vdim).  release() zeroes the states; cache rows need no clearing, a sequence only reads positions it wrote.
//
// Precision: the residual stream, norms, rotation angles, scores, softmax, router, the recurrence with its state, gates and every sum are
// fp32 in both modes.  XALM_PRECISION_BF16 keeps matrices and the latent cache in bf16 and sends dense products of long passes through
// the tcgen05 GEMM (fp16 operands, fp32 accumulation); XALM_PRECISION_F32 widens both and uses the fp32 FMA kernels only.
#include "seq_family.cuh"

#include "seq_latent.cuh"
#include "seq_moe.cuh"

namespace xalm {
namespace {

using namespace mix;
using namespace seq;

enum { MIX_LATENT = 0, MIX_LATENT_GATED = 1, MIX_RETENTION = 2 };
enum { FF_NONE = 0, FF_DENSE = 1, FF_MOE = 2 };

struct Layer {
	int mixer = MIX_LATENT, ff_kind = FF_NONE;
	int H = 0, d = 0, dv = 0;
	// latent attention
	LatentWeights lat;
	int kv_from = -1;
	LatentCache cache; // this layer's rows, or the rows of the layer it reads
	// retention
	int rot_dims = 0;
	std::vector<float> decay_host;
	float *decay = nullptr, *state = nullptr;
	std::vector<float> freq_host;
	float* freq = nullptr;
	int off_a = 0, off_b = 0, off_g = 0, n_in = 0; // columns of the stacked input projection [q | k | v | g]
	// feed-forward
	int ff = 0; // dense
	MoeWeights moe;
	float limit = 0.f;
	void *w_in = nullptr, *w_o = nullptr, *w_up = nullptr, *w_down = nullptr;
	WMat m_in, m_o, m_up, m_down;
	TcWeight t_in, t_o, t_up, t_down;
	float *norm1 = nullptr, *norm2 = nullptr;
};

struct DuletarModel : SeqModel {
	float embed_scale = 1.f, logit_cap = 0.f;
	std::vector<Layer> layers;
	// one pass
	float *x = nullptr, *hn = nullptr, *proj = nullptr, *att = nullptr, *ffh = nullptr;
	int proj_ld = 4;
	LatentBuffers lat;
	AttnParts parts;
	MoeBuffers moe;
};
typedef DuletarModel Du;

// ---- config.json ------------------------------------------------------------------------------------------------------------------
int parse_config(SeqModel* sm, const char* json) {
	Du* m = static_cast<Du*>(sm);
	try {
		const xjson::Value c = xjson::Parser::parse(json, strlen(json));
		m->vocab = geti(c, "vocab");
		m->width = geti(c, "width");
		if (const xjson::Value* nv = c.find("norm"))
			if (const xjson::Value* e = nv->find("eps")) m->eps = (float) e->num;
		if (const xjson::Value* ev = c.find("embedding"); ev && ev->kind == xjson::Value::Obj && ev->contains("scale")) m->embed_scale = (float) getf(*ev, "scale");
		if (const xjson::Value* lc = c.find("logit_softcap"); lc && lc->kind == xjson::Value::Number) m->logit_cap = (float) lc->num;
		if (m->vocab <= 0 || m->width <= 0) return set_error(XALM_ERR_INVALID, "config: vocab / width must be positive");
		const int W = m->width;
		expect(m, "embed", {m->vocab, W}, true);
		const xjson::Value& layers = c.at("layers");
		if (layers.kind != xjson::Value::Array || layers.arr.empty()) return set_error(XALM_ERR_INVALID, "config: no layers");
		for (size_t li = 0; li < layers.arr.size(); li++) {
			const xjson::Value& lv = layers.arr[li];
			const std::string type = lv.at("type").str;
			Layer L;
			if (type == "latent_attention") L.mixer = MIX_LATENT;
			else if (type == "latent_attention_2") L.mixer = MIX_LATENT_GATED;
			else if (type == "retention") L.mixer = MIX_RETENTION;
			else return set_error(XALM_ERR_UNSUPPORTED, "config: layer %zu has mixer type '%s' (this family runs 'latent_attention', 'latent_attention_2' and 'retention')", li, type.c_str());
			const xjson::Value& mx = lv.at("mixer");
			L.H = geti(mx, "heads");
			L.d = geti(mx, "dim");
			L.dv = mx.contains("vdim") ? geti(mx, "vdim") : L.d;
			if (L.H <= 0 || L.d <= 0 || L.dv <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: bad mixer sizes", li);
			const std::string p = "l" + std::to_string(li) + ".";
			const int H = L.H, d = L.d, dv = L.dv;
			const xjson::Value* rt = mx.find("rot");
			if (rt && rt->kind != xjson::Value::Obj) rt = nullptr;
			expect(m, p + "norm1", {W}, false);
			if (L.mixer == MIX_RETENTION) {
				const xjson::Value& dc = mx.at("decay");
				if (dc.kind != xjson::Value::Array || (int) dc.arr.size() != H) return set_error(XALM_ERR_INVALID, "config: layer %zu: 'decay' lists one value per head", li);
				for (const xjson::Value& v : dc.arr) L.decay_host.push_back((float) v.num);
				if (rt) {
					L.rot_dims = geti(*rt, "dims");
					if (L.rot_dims < 0 || L.rot_dims > d || L.rot_dims % 2) return set_error(XALM_ERR_INVALID, "config: layer %zu: %d rotary dimensions in a head of %d", li, L.rot_dims, d);
					if (L.rot_dims) L.freq_host = rotary_frequencies(getf(*rt, "base"), L.rot_dims);
				}
				expect(m, p + "mix.q", {H * d, W}, true);
				expect(m, p + "mix.k", {H * d, W}, true);
				expect(m, p + "mix.v", {H * dv, W}, true);
				expect(m, p + "mix.g", {H * dv, W}, true);
			} else {
				LatentWeights& A = L.lat;
				A.H = H; A.d = d; A.dv = dv;
				A.R = geti(mx, "kv_rank");
				A.Rq = geti(mx, "q_rank");
				A.gate = L.mixer == MIX_LATENT_GATED ? LATENT_GATE_COLUMNS : LATENT_GATE_NONE;
				A.scale = mx.contains("scale") ? (float) getf(mx, "scale") : 1.f / sqrtf((float) d);
				if (L.mixer == MIX_LATENT) {
					A.r = mx.contains("rot_dim") ? geti(mx, "rot_dim") : 0;
					if (A.r < 0 || A.r % 2) return set_error(XALM_ERR_INVALID, "config: layer %zu: rot_dim %d", li, A.r);
					if (A.r) {
						if (!rt) return set_error(XALM_ERR_INVALID, "config: layer %zu: rot_dim without 'rot'", li);
						const int dims = rt->contains("dims") ? geti(*rt, "dims") : A.r;
						if (dims != A.r) return set_error(XALM_ERR_INVALID, "config: layer %zu: rot.dims %d differs from rot_dim %d", li, dims, A.r);
						A.freq_host = rotary_frequencies(getf(*rt, "base"), A.r);
					}
				}
				if (A.R <= 0 || A.Rq <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: latent sizes", li);
				if (const xjson::Value* kf = mx.find("kv_from"); kf && kf->kind == xjson::Value::Number) {
					if (L.mixer != MIX_LATENT_GATED) return set_error(XALM_ERR_UNSUPPORTED, "config: layer %zu: kv_from on a rotary latent attention", li);
					L.kv_from = (int) kf->num;
					if (L.kv_from < 0 || L.kv_from >= (int) li) return set_error(XALM_ERR_INVALID, "config: layer %zu: kv_from %d is not an earlier layer", li, L.kv_from);
					const Layer& J = m->layers[(size_t) L.kv_from];
					if (J.mixer == MIX_RETENTION || J.kv_from >= 0 || J.lat.R != A.R)
						return set_error(XALM_ERR_INVALID, "config: layer %zu: layer %d has no latents of %d of its own", li, L.kv_from, A.R);
				}
				A.own_cache = L.kv_from < 0;
				latent_expect(m, p + "mix.", A);
			}
			expect(m, p + "mix.o", {W, H * dv}, true);
			const xjson::Value* mlp = lv.find("mlp");
			if (mlp && mlp->kind == xjson::Value::Obj) {
				const std::string kind = mlp->contains("kind") ? mlp->at("kind").str : "dense";
				expect(m, p + "norm2", {W}, false);
				if (kind == "dense") {
					L.ff_kind = FF_DENSE;
					L.ff = geti(*mlp, "ff");
					if (L.ff <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: ff", li);
					expect(m, p + "mlp.up", {L.ff, W}, true);
					expect(m, p + "mlp.down", {W, L.ff}, true);
				} else if (kind == "moe") {
					L.ff_kind = FF_MOE;
					const xjson::Value& ex = mlp->at("expert");
					L.moe.ff = geti(ex, "ff");
					L.limit = (float) getf(ex, "limit");
					const xjson::Value& r = mlp->at("router");
					L.moe.E = geti(r, "experts");
					L.moe.top = geti(r, "top");
					if (const xjson::Value* g = r.find("groups"); g && g->kind == xjson::Value::Obj) {
						L.moe.n_groups = geti(*g, "count");
						L.moe.keep_groups = geti(*g, "keep");
					}
					if (L.moe.ff <= 0 || L.moe.E <= 0 || L.moe.top <= 0 || L.moe.top > L.moe.E) return set_error(XALM_ERR_INVALID, "config: layer %zu: %d of %d experts of %d", li, L.moe.top, L.moe.E, L.moe.ff);
					if (L.moe.n_groups > 1 && (L.moe.E % L.moe.n_groups || L.moe.keep_groups <= 0 || L.moe.keep_groups > L.moe.n_groups || L.moe.keep_groups * (L.moe.E / L.moe.n_groups) < L.moe.top))
						return set_error(XALM_ERR_INVALID, "config: layer %zu: %d expert groups with %d kept cannot hold %d of %d experts", li, L.moe.n_groups, L.moe.keep_groups, L.moe.top, L.moe.E);
					moe_expect(m, p + "mlp.", L.moe.E, L.moe.ff, true);
					expect(m, p + "mlp.router", {L.moe.E, W}, true);
				} else return set_error(XALM_ERR_UNSUPPORTED, "config: layer %zu has feed-forward kind '%s'", li, kind.c_str());
			}
			m->layers.push_back(std::move(L));
		}
		m->n_layers = (int) m->layers.size();
		expect(m, "final.norm", {W}, false);
		expect(m, "head", {m->vocab, W}, true);
	} catch (const std::exception& e) {
		return set_error(XALM_ERR_INVALID, "config.json: %s", e.what());
	}
	return XALM_OK;
}

// ---- the kernels of one pass ----------------------------------------------------------------------------------------------------------
RowsEpi residual_epi(Du* m) { // x <- x + product: the single-stream case of the hyper-connection write
	RowsEpi e;
	e.kind = EPI_HC;
	e.xs = m->x;
	e.S = 1;
	e.stream_stride = (size_t) m->chunk * m->width;
	return e;
}

int enqueue_retention(Du* m, const Layer& L, int n, int* nl) {
	cudaStream_t s = m->stream;
	const int H = L.H, d = L.d, dv = L.dv;
	if (L.rot_dims) {
		RopeHeadsArgs ra = {};
		ra.src = m->proj; ra.dst = m->proj; ra.lds = ra.ldd = m->proj_ld; ra.src_off = ra.dst_off = 0; ra.src_stride = ra.dst_stride = d;
		ra.heads = 2 * H; ra.n = d; ra.rot_half = L.rot_dims / 2; ra.freq = L.freq; ra.step = m->d_step; // q heads, then k heads
		XALM_TRY(launch_rope_heads(ra, n, s));
		(*nl)++;
	}
	Hgrn2Args ha = {};
	ha.proj = m->proj; ha.ld = m->proj_ld; ha.q_off = 0; ha.k_off = L.off_a; ha.v_off = L.off_b;
	ha.H = H; ha.d = d; ha.dv = dv;
	ha.decay = L.decay; ha.k_scale = 1.f / sqrtf((float) d);
	ha.norm_plain = 1; ha.eps = m->eps;
	ha.gate = m->proj; ha.ldg = m->proj_ld; ha.g_off = L.off_g;
	ha.state = L.state; ha.step = m->d_step; ha.out = m->att; ha.max_rows = m->chunk;
	XALM_TRY(launch_hgrn2(ha, s));
	(*nl)++;
	return XALM_OK;
}

int enqueue_experts(Du* m, const Layer& L, int n, int* nl) {
	MoeRouteArgs ra = {};
	ra.score_kind = MOE_SCORE_SOFTMAX; ra.group_kind = MOE_GROUP_MAX; ra.renormalise = 1; ra.renorm_eps = 1e-20f;
	RowsEpi eg;
	eg.kind = EPI_GLU; eg.glu_act = GLU_CLAMPED; eg.limit = L.limit; eg.alpha = 1.702f;
	MoeCombineArgs ca = {};
	ca.x_in = m->x; ca.x_out = m->x;
	XALM_TRY(moe_experts(m, L.moe, m->moe, m->hn, n, ra, eg, &ca, nl));
	XALM_TRY(launch_moe_combine(ca, n, m->stream));
	(*nl)++;
	return XALM_OK;
}

int enqueue_pass(SeqModel* sm, int n, int want, int* nl) {
	Du* m = static_cast<Du*>(sm);
	cudaStream_t s = m->stream;
	const int W = m->width;
	const size_t hs = (size_t) m->chunk * W;
	if (m->w_bf16) embed_streams_kernel<__nv_bfloat16><<<n, norm_threads(W), 0, s>>>((const __nv_bfloat16*) m->embed, m->d_tokens, W, 1, hs, m->x, m->embed_scale);
	else embed_streams_kernel<float><<<n, norm_threads(W), 0, s>>>((const float*) m->embed, m->d_tokens, W, 1, hs, m->x, m->embed_scale);
	XALM_SEQ_LAUNCH_CHECK("embed");
	for (size_t li = 0; li < m->layers.size(); li++) {
		const Layer& L = m->layers[li];
		XALM_TRY(launch_hc_norm(m->x, 1, hs, nullptr, L.norm1, 0, m->eps, W, m->hn, nullptr, n, s));
		(*nl)++;
		RowsEpi est;
		est.kind = EPI_STORE; est.out = m->proj; est.ldo = m->proj_ld;
		if (L.mixer == MIX_RETENTION) {
			XALM_TRY(rows_product(m, m->hn, W, L.w_in, &L.t_in, n, L.n_in, W, est, nl));
			XALM_TRY(enqueue_retention(m, L, n, nl));
		} else {
			XALM_TRY(rows_product(m, m->hn, W, L.lat.w_in, &L.lat.t_in, n, L.lat.n_in, W, est, nl));
			XALM_TRY(latent_attention(m, L.lat, L.cache, m->lat, m->parts, m->proj, m->proj_ld, m->att, n, nl));
		}
		XALM_TRY(rows_product(m, m->att, L.H * L.dv, L.w_o, &L.t_o, n, W, L.H * L.dv, residual_epi(m), nl));
		if (L.ff_kind != FF_NONE) {
			XALM_TRY(launch_hc_norm(m->x, 1, hs, nullptr, L.norm2, 0, m->eps, W, m->hn, nullptr, n, s));
			(*nl)++;
		}
		if (L.ff_kind == FF_DENSE) {
			RowsEpi ea;
			ea.kind = EPI_ACT; ea.act = ACT_RELU_SQUARED; ea.out = m->ffh; ea.ldo = L.ff;
			XALM_TRY(rows_product(m, m->hn, W, L.w_up, &L.t_up, n, L.ff, W, ea, nl));
			XALM_TRY(rows_product(m, m->ffh, L.ff, L.w_down, &L.t_down, n, W, L.ff, residual_epi(m), nl));
		} else if (L.ff_kind == FF_MOE) XALM_TRY(enqueue_experts(m, L, n, nl));
		if (m->keep_layers) XALM_CUDA_CHECK(cudaMemcpyAsync(m->layer_sums + li * hs, m->x, (size_t) n * W * 4, cudaMemcpyDeviceToDevice, s));
	}
	if (want) {
		const int rows = want == 2 ? n : 1, first = want == 2 ? 0 : n - 1;
		XALM_TRY(launch_hc_norm(m->x + (size_t) first * W, 1, hs, nullptr, m->final_norm, 0, m->eps, W, m->hn, nullptr, rows, s));
		(*nl)++;
		RowsEpi eh;
		eh.kind = EPI_STORE; eh.out = m->logits; eh.ldo = m->vocab; eh.cap = m->logit_cap;
		XALM_TRY(rows_product(m, m->hn, W, m->w_head, &m->t_head, rows, m->vocab, W, eh, nl));
	}
	return XALM_OK;
}

// ---- device layouts, cache, state, pass buffers ---------------------------------------------------------------------------------------
int finalize(SeqModel* sm) {
	Du* m = static_cast<Du*>(sm);
	const int W = m->width;
	const size_t C = (size_t) m->chunk;
	auto T = [&](const std::string& n) { return tensor_or_null(m, n); };
	size_t max_in = 4, max_att = 1, max_ff = 1;
	for (size_t li = 0; li < m->layers.size(); li++) {
		Layer& L = m->layers[li];
		const std::string p = "l" + std::to_string(li) + ".";
		const int H = L.H, d = L.d, dv = L.dv;
		XALM_TRY(upload_vec(m, p + "norm1", &L.norm1));
		if (!L.freq_host.empty()) XALM_TRY(upload_floats(m, L.freq_host.data(), L.freq_host.size(), &L.freq));
		if (L.mixer == MIX_RETENTION) {
			L.off_a = H * d; L.off_b = 2 * H * d; L.off_g = L.off_b + H * dv; L.n_in = L.off_g + H * dv;
			XALM_TRY(upload_rows(m, {T(p + "mix.q"), T(p + "mix.k"), T(p + "mix.v"), T(p + "mix.g")}, W, false, &L.w_in, &L.m_in));
			XALM_TRY(upload_floats(m, L.decay_host.data(), L.decay_host.size(), &L.decay));
			XALM_TRY(dev_alloc(m, &L.state, (size_t) H * d * dv, true));
			if (!hgrn2_cols_ok(d, dv, m->chunk) && hgrn2_smem_bytes(d, dv) > 200 * 1024)
				return set_error(XALM_ERR_UNSUPPORTED, "layer %zu: a retention state of %d x %d per head", li, d, dv);
			XALM_TRY(hgrn2_prepare(d, dv));
		} else {
			XALM_TRY(latent_upload(m, p + "mix.", li, &L.lat, &m->lat, &m->parts));
			if (L.kv_from < 0) XALM_TRY(latent_cache_alloc(m, L.lat, &L.cache));
			else L.cache = m->layers[(size_t) L.kv_from].cache;
			max_in = std::max(max_in, (size_t) L.lat.n_in);
		}
		XALM_TRY(upload_rows(m, {T(p + "mix.o")}, H * dv, false, &L.w_o, &L.m_o));
		max_in = std::max(max_in, (size_t) L.n_in);
		max_att = std::max(max_att, (size_t) H * dv);
		if (L.ff_kind != FF_NONE) XALM_TRY(upload_vec(m, p + "norm2", &L.norm2));
		if (L.ff_kind == FF_DENSE) {
			XALM_TRY(upload_rows(m, {T(p + "mlp.up")}, W, false, &L.w_up, &L.m_up));
			XALM_TRY(upload_rows(m, {T(p + "mlp.down")}, L.ff, false, &L.w_down, &L.m_down));
			max_ff = std::max(max_ff, (size_t) L.ff);
		} else if (L.ff_kind == FF_MOE) {
			XALM_TRY(moe_upload(m, p + "mlp.", true, &L.moe, &m->moe));
		}
	}
	XALM_TRY(hc_norm_prepare(W));
	for (Layer& L : m->layers) {
		if (L.mixer == MIX_RETENTION) XALM_TRY(tc_register(m, L.m_in, &L.t_in));
		else XALM_TRY(latent_tc_register(m, &L.lat));
		XALM_TRY(tc_register(m, L.m_o, &L.t_o));
		if (L.ff_kind == FF_DENSE) {
			XALM_TRY(tc_register(m, L.m_up, &L.t_up));
			XALM_TRY(tc_register(m, L.m_down, &L.t_down));
		}
		if (L.ff_kind == FF_MOE) XALM_TRY(moe_tc_register(m, &L.moe, &m->moe));
	}
	m->proj_ld = (int) ((max_in + 3) / 4 * 4);
	XALM_TRY(dev_alloc(m, &m->x, C * W));
	XALM_TRY(dev_alloc(m, &m->hn, C * W));
	XALM_TRY(dev_alloc(m, &m->proj, C * m->proj_ld));
	XALM_TRY(latent_alloc(m, &m->lat));
	XALM_TRY(dev_alloc(m, &m->att, C * max_att));
	XALM_TRY(dev_alloc(m, &m->ffh, C * max_ff));
	XALM_TRY(attn_parts_alloc(m, &m->parts));
	return moe_alloc(m, &m->moe);
}

int release(SeqModel* sm) {
	Du* m = static_cast<Du*>(sm);
	for (Layer& L : m->layers)
		if (L.mixer == MIX_RETENTION) XALM_CUDA_CHECK(cudaMemsetAsync(L.state, 0, (size_t) L.H * L.d * L.dv * 4, m->stream));
	return XALM_OK;
}

// beyond the matrices: the visible cache rows, the recurrent state read and written; of a mixture only the chosen experts are read
long long active_bytes(SeqModel* sm, long long pos) {
	Du* m = static_cast<Du*>(sm);
	long long b = 0;
	const long long kelem = m->precision == XALM_PRECISION_F32 ? 4 : 2, welem = m->w_bf16 ? 2 : 4;
	for (const Layer& L : m->layers) {
		if (L.mixer == MIX_RETENTION) b += 2ll * L.H * L.d * L.dv * 4;
		else b += (pos + 1) * (L.lat.R + L.lat.r) * kelem;
		if (L.ff_kind == FF_MOE) b -= (long long) (L.moe.E - L.moe.top) * 3 * L.moe.ff * m->width * welem;
	}
	return b;
}

bool state_buffer(SeqModel* sm, int layer, const float** src, size_t* count) {
	Du* m = static_cast<Du*>(sm);
	const Layer& L = m->layers[(size_t) layer];
	if (L.mixer != MIX_RETENTION) return false;
	*src = L.state;
	*count = (size_t) L.H * L.d * L.dv;
	return true;
}

void destroy(SeqModel* sm) {
	Du* m = static_cast<Du*>(sm);
	for (Layer& L : m->layers) {
		for (TcWeight* t : {&L.t_in, &L.t_o, &L.t_up, &L.t_down}) tc_weight_free(t);
		latent_free(&L.lat);
		moe_free(&L.moe);
	}
	delete m;
}

const SeqHooks duletar_hooks = {parse_config, finalize, enqueue_pass, release, active_bytes, state_buffer, destroy};
extern const ModelFamily duletar_family;
int create(const char* json, int device, int max_tokens, int precision, xalm_cuda_model** out) {
	return seq_create<Du>(&duletar_family, &duletar_hooks, json, device, max_tokens, precision, out);
}
const ModelFamily duletar_family = seq_family_table("Duletar", create);
const FamilyRegistrar duletar_registrar(&duletar_family);

} // namespace
} // namespace xalm
