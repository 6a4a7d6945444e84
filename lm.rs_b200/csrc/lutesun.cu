// lutesun.cu -- the Lutesun architecture (arch.h): a decoder whose sublayers read the residual stream itself and whose outputs are
// RMS-normed (weight stored around zero) and added,
//     x0 = scale * embed[token];   x <- x + rms(mixer(x)) (1 + n1);   x <- x + rms(ff(x)) (1 + n2)       (a layer may have no ff)
// Every mixer is windowed attention through a latent (latent_mixer.cuh), in two forms listed per layer in config.json "layers":
//   "latent_attention"    queries straight from x, neighbouring dimensions rotated in pairs
//   "latent_attention_2"  queries through a normed latent, rotation in halves, one sigmoid output gate per head
// and two kinds of feed-forward: "dense" (W_down relu(W_up x + b)^2 + b) and "moe" (softmax router over experts and identity
// experts, choice by score + correction inside the best groups of neighbouring outputs, weights renormalised over the chosen and
// scaled; experts are SiLU GLUs; an optional shared expert times the sigmoid of one logit per token).  logits = embed (rms(x) (1 + w))
// with the unscaled embedding table.  Everything model-specific comes from config.json and the tensor shapes; the kernels are the
// generic ones of dense_ops.cuh / mixer_ops.cuh / moe_ops.cuh / dense_gemm.cuh, the step / chunking / graph machinery is
// DenseModel's.  Caches are addressed by position; no layer carries other state, so a step may start at any cached position.
#include "latent_mixer.cuh"
#include "moe_ops.cuh"

namespace lmrs {
namespace {

enum LuFf { LU_FF_NONE = 0, LU_FF_DENSE = 1, LU_FF_MOE = 2 };

struct LuFfCfg {
    int kind = LU_FF_NONE;
    int ff = 0;                      // dense: hidden size; moe: hidden size of one expert
    int E = 0, I = 0, top = 0;       // experts with matrices, identity experts, choices per token
    int groups = 1, keep = 1;
    float scale = 1.0f;
    int shared_ff = 0;
};

template <typename AT, typename WT> class LutesunModel : public LatentModel<AT, WT> {
  public:
    typedef LatentModel<AT, WT> B;
    using B::load_vec; using B::load_stack; using B::load_stack_f32; using B::load_offset_vec; using B::error; using B::launches; using B::info; using B::d_logits;
    using B::width; using B::vocab; using B::max_tokens; using B::sms; using B::d_tokens; using B::cap; using B::x; using B::hn; using B::d_rows; using B::pdl_now;
    using B::dalloc; using B::dfree; using B::check_launch; using B::launch_k; using B::drop_graphs;

    struct Layer {
        typename B::Latent mix;
        LuFfCfg f;
        float *norm1 = nullptr, *norm2 = nullptr;   // 1 + w
        WT* wo = nullptr;
        WT *wgate = nullptr, *wup = nullptr, *wdown = nullptr;   // dense: up [ff][width], down [width][ff]; moe: the experts' back to back
        float *bup = nullptr, *bdown = nullptr;                  // dense
        float *router = nullptr, *correction = nullptr;          // router rows, then the shared expert's gate row
        WT *sgate = nullptr, *sup = nullptr, *sdown = nullptr;   // shared expert
    };
    std::vector<Layer> layers;
    WT* embed = nullptr;
    float* final_norm = nullptr;   // 1 + w
    float embed_scale = 1.0f;
    // scratch for `cap` rows
    AT *h = nullptr, *act = nullptr, *act_sh = nullptr, *xg = nullptr;
    float *proj = nullptr, *yf = nullptr, *ye = nullptr, *ysh = nullptr, *rz = nullptr, *wts = nullptr;
    int *eidx = nullptr, *slot = nullptr, *row_of = nullptr, *grp = nullptr;
    int max_proj = 0, max_act = 0, max_eff = 0, max_top = 0, max_E = 0, max_shared = 0;

    size_t n_layers() const override { return layers.size(); }

    // ---- configuration ---------------------------------------------------------------------------------------------------
    int parse_layer(const Json& jl, size_t li, Layer& L) {
        const std::string type = jl.at("type").str, where = "config.json layers[" + std::to_string(li) + "]";
        if (type != "latent_attention" && type != "latent_attention_2") { error = where + ": unknown layer type '" + type + "'"; return 1; }
        const Json& m = jl.at("mixer");
        LatentCfg& c = L.mix.c;
        if (this->parse_latent(m, where, c)) return 1;
        if (type == "latent_attention_2") {
            c.rq = (int)m.at("q_rank").number(0);
            c.gate = c.halves = true;
            if (c.rq <= 0) { error = where + ": q_rank is required"; return 1; }
        }
        if (c.rot_dims > 0) {
            const double base = m.at("rot").at("base").number(10000.0);
            for (int i = 0; i < c.rot_dims / 2; i++) c.rot_f.push_back(pow(base, -2.0 * (double)i / (double)c.rot_dims));
            char key[160];
            snprintf(key, sizeof key, "plain/%d/%.17g", c.rot_dims, base);
            c.rot_key = key;
        }
        if (!jl.has("mlp") || !jl.at("mlp").is_obj()) return 0;
        const Json& f = jl.at("mlp");
        LuFfCfg& o = L.f;
        const std::string kind = f.has("kind") ? f.at("kind").str : "dense";
        if (kind == "dense") {
            o.kind = LU_FF_DENSE;
            o.ff = (int)f.at("ff").number(0);
            if (o.ff <= 0) { error = where + ": mlp.ff is required"; return 1; }
        } else if (kind == "moe") {
            o.kind = LU_FF_MOE;
            o.ff = (int)f.at("expert").at("ff").number(0);
            const Json& r = f.at("router");
            o.E = (int)r.at("experts").number(0); o.top = (int)r.at("top").number(0);
            o.I = r.has("identity") ? (int)r.at("identity").number(0) : 0;
            o.scale = r.has("scale") ? (float)r.at("scale").number(1.0) : 1.0f;
            if (r.has("groups") && r.at("groups").is_obj()) { o.groups = (int)r.at("groups").at("count").number(1); o.keep = (int)r.at("groups").at("keep").number(1); }
            if (f.has("shared") && f.at("shared").is_obj()) o.shared_ff = (int)f.at("shared").at("ff").number(0);
            const int n = o.E + o.I;
            if (o.E <= 0 || o.I < 0 || o.ff <= 0 || o.top <= 0 || n > 4096 || o.shared_ff < 0) { error = where + ": bad expert geometry"; return 1; }
            if (o.groups <= 0 || n % o.groups != 0 || o.keep <= 0 || o.keep > o.groups) { error = where + ": router.groups must divide the experts and keep 1 .. count of them"; return 1; }
            if (o.top > o.keep * (n / o.groups)) { error = where + ": router.top exceeds the experts of the kept groups"; return 1; }
        } else { error = where + ": unknown mlp kind '" + kind + "'"; return 1; }
        return 0;
    }

    // ---- weights -----------------------------------------------------------------------------------------------------------
    int load_ff(const SafeTensors& st, const std::string& p, Layer& L) {
        const LuFfCfg& f = L.f;
        if (f.kind == LU_FF_DENSE) {
            max_act = std::max(max_act, f.ff);
            return load_stack(st, {{p + "up", f.ff}}, width, &L.wup, nullptr) || load_vec(st, p + "up.b", f.ff, &L.bup) ||
                   load_stack(st, {{p + "down", width}}, f.ff, &L.wdown, nullptr) || load_vec(st, p + "down.b", width, &L.bdown);
        }
        std::vector<std::pair<std::string, int>> rows = {{p + "router", f.E + f.I}}, gs, us, ds;
        for (int e = 0; e < f.E; e++) {
            const std::string pe = p + "e" + std::to_string(e) + ".";
            gs.push_back({pe + "gate", f.ff}); us.push_back({pe + "up", f.ff}); ds.push_back({pe + "down", width});
        }
        if (load_stack(st, gs, width, &L.wgate, nullptr) || load_stack(st, us, width, &L.wup, nullptr) || load_stack(st, ds, f.ff, &L.wdown, nullptr)) return 1;
        if (f.shared_ff > 0) {
            rows.push_back({p + "shared.sg", 1});
            if (load_stack(st, {{p + "shared.gate", f.shared_ff}}, width, &L.sgate, nullptr) || load_stack(st, {{p + "shared.up", f.shared_ff}}, width, &L.sup, nullptr) ||
                load_stack(st, {{p + "shared.down", width}}, f.shared_ff, &L.sdown, nullptr))
                return 1;
        }
        if (load_stack_f32(st, rows, width, &L.router)) return 1;
        if (st.find(p + "correction") && load_vec(st, p + "correction", f.E + f.I, &L.correction)) return 1;
        max_top = std::max(max_top, f.top); max_eff = std::max(max_eff, f.ff); max_E = std::max(max_E, f.E + f.I); max_shared = std::max(max_shared, f.shared_ff);
        return 0;
    }

    int load(const std::string& dir, const Json& cfg, const ArchOptions& opt) {
        sms = opt.sms;
        B::gemm_ctx.sms = opt.sms;
        width = (int)cfg.at("width").number(0);
        vocab = (int)cfg.at("vocab").number(0);
        if (width <= 0 || vocab <= 0) { error = "config.json: width and vocab are required"; return 1; }
        const float eps = (float)cfg.at("norm").at("eps").number(1e-6);
        embed_scale = cfg.has("embedding") && cfg.at("embedding").is_obj() ? (float)cfg.at("embedding").at("scale").number(1.0) : 1.0f;
        max_tokens = opt.max_tokens ? opt.max_tokens : 4096u;
        const Json& jl = cfg.at("layers");
        if (jl.kind != Json::ARR || jl.arr.empty()) { error = "config.json: 'layers' must be a non-empty list"; return 1; }
        SafeTensors st;
        if (!st.open(dir + "/model.safetensors", error)) return 1;
        if (load_stack(st, {{"embed", vocab}}, width, &embed, nullptr) || load_offset_vec(st, "final.norm", width, &final_norm)) return 1;
        layers.resize(jl.arr.size());
        for (size_t li = 0; li < layers.size(); li++) {
            Layer& L = layers[li];
            if (parse_layer(jl.arr[li], li, L)) return 1;
            const std::string p = "l" + std::to_string(li) + ".";
            const LatentCfg& c = L.mix.c;
            if (load_offset_vec(st, p + "norm1", width, &L.norm1) || this->load_latent(st, p + "mix.", L.mix) ||
                load_stack(st, {{p + "mix.o", width}}, c.H * c.dv, &L.wo, nullptr))
                return 1;
            max_proj = std::max(max_proj, L.mix.in_rows);
            if (L.f.kind != LU_FF_NONE && (load_offset_vec(st, p + "norm2", width, &L.norm2) || load_ff(st, p + "mlp.", L))) return 1;
        }
        if (dalloc(&d_tokens, (size_t)max_tokens) || dalloc(&d_logits, (size_t)vocab)) return 1;
        GCK(cudaMemset(d_tokens, 0, (size_t)max_tokens * 4));
        info.architecture = "Lutesun";
        info.model_type = 8;
        info.vocab = (uint32_t)vocab; info.width = (uint32_t)width; info.n_layers = (uint32_t)layers.size(); info.max_tokens = max_tokens;
        info.heads = (uint32_t)layers[0].mix.c.H; info.kv_heads = 1; info.head_dim = (uint32_t)layers[0].mix.c.dn;
        info.ff = (uint32_t)layers[0].f.ff; info.dtype = opt.dtype; info.eps = eps;
        return ensure_scratch(1);
    }

    int ensure_scratch(size_t rows) override {
        if (rows <= cap) return 0;
        drop_graphs();   // captured launches point into the old scratch
        for (void* p : {(void*)x, (void*)hn, (void*)d_rows, (void*)h, (void*)act, (void*)act_sh, (void*)xg, (void*)proj, (void*)yf, (void*)ye, (void*)ysh, (void*)rz,
                        (void*)wts, (void*)eidx, (void*)slot, (void*)row_of, (void*)grp})
            dfree(p);
        x = nullptr; hn = nullptr; d_rows = nullptr; h = nullptr; act = nullptr; act_sh = nullptr; xg = nullptr; proj = nullptr; yf = nullptr; ye = nullptr;
        ysh = nullptr; rz = nullptr; wts = nullptr; eidx = nullptr; slot = nullptr; row_of = nullptr; grp = nullptr;
        cap = 0;
        const size_t pairs = rows * max_top;
        if (dalloc(&x, rows * width) || dalloc(&hn, rows * width) || dalloc(&d_rows, rows) || dalloc(&h, rows * width) ||
            dalloc(&act, std::max(rows * max_act, pairs * max_eff)) || dalloc(&act_sh, rows * max_shared) || dalloc(&xg, pairs * width) ||
            dalloc(&proj, rows * max_proj) || dalloc(&yf, rows * width) || dalloc(&ye, pairs * width) || dalloc(&ysh, max_shared > 0 ? rows * width : 0) ||
            dalloc(&rz, rows * (max_E + 1)) || dalloc(&wts, pairs) || dalloc(&eidx, pairs) || dalloc(&slot, pairs) || dalloc(&row_of, pairs) ||
            dalloc(&grp, (size_t)max_E + 1) || this->ensure_latent_scratch(rows))
            return 1;
        cap = rows;
        return 0;
    }

    // ---- the layers -----------------------------------------------------------------------------------------------------------
    int one_row_threads() const { return std::min(1024, (width + 31) / 32 * 32); }
    // a sublayer's last product, its norm, the residual, and x again in the operand type for the next sublayer
    int sublayer_out(cudaStream_t st, int T, const AT* a, int K, const WT* w, const float* bias, const float* nw) {
        EpiParams<AT> e{}; e.out = yf; e.ldo = width; e.scale = 1.0f; e.bias = bias;
        if (this->template matmul<EPI_STORE>(st, T, a, K, w, nullptr, K, width, e)) return 1;
        ResNormRowsParams<AT> p{};
        p.y = yf; p.ldy = width; p.wb = nw; p.x = x; p.ldx = width; p.n = width; p.eps = info.eps; p.h = h; p.ldh = width;
        if (T == 1) return launch_k("resnorm_rows_kernel", st, pdl_now, resnorm_rows_kernel<AT, true>, dim3(1), dim3(one_row_threads()), 0, p);
        return launch_k("resnorm_rows_kernel", st, pdl_now, resnorm_rows_kernel<AT, false>, dim3(T), dim3(256), 0, p);
    }
    int mixer(cudaStream_t st, const Layer& L, int T, const PosSrc& ps, uint32_t pos_hint) {
        EpiParams<AT> e{}; e.out = proj; e.ldo = L.mix.in_rows; e.scale = 1.0f;
        if (this->template matmul<EPI_STORE>(st, T, h, width, L.mix.w_in, nullptr, width, L.mix.in_rows, e)) return 1;
        const AT* heads = nullptr;
        if (this->mixer_latent(st, L.mix, T, ps, pos_hint, proj, &heads)) return 1;
        return sublayer_out(st, T, heads, L.mix.c.H * L.mix.c.dv, L.wo, nullptr, L.norm1);
    }
    int ff_dense(cudaStream_t st, const Layer& L, int T) {
        EpiParams<AT> eu{}; eu.act = act; eu.lda = L.f.ff; eu.act_kind = ACT_RELU2; eu.bias = L.bup;
        if (this->template matmul<EPI_ACT>(st, T, h, width, L.wup, nullptr, width, L.f.ff, eu)) return 1;
        return sublayer_out(st, T, act, L.f.ff, L.wdown, L.bdown, L.norm2);
    }
    int ff_moe(cudaStream_t st, const Layer& L, int T) {
        const LuFfCfg& f = L.f;
        const int n_out = f.E + f.I;
        const bool sh = f.shared_ff > 0;
        MoeRouterParams<AT> rp{};
        rp.h = h; rp.ld = width; rp.router = L.router; rp.correction = L.correction; rp.E = n_out; rp.extra = sh ? 1 : 0; rp.top = f.top; rp.width = width;
        rp.groups = f.groups; rp.keep = f.keep; rp.softmax = 1; rp.scale = f.scale; rp.z = rz; rp.idx = eidx; rp.wts = wts;
        if (launch_k("moe_logits_kernel", st, pdl_now, moe_logits_kernel<AT>, dim3(T, (n_out + rp.extra + 3) / 4), dim3(128), 0, rp)) return 1;
        if (launch_k("moe_topk_kernel", st, pdl_now, moe_topk_kernel<AT>, dim3(T), dim3(32), ((size_t)2 * n_out + f.groups) * 4, rp)) return 1;
        MoeCombineResNormParams<AT> np{};
        MoeCombineParams& cp = np.c;
        cp.y = ye; cp.wts = wts; cp.top = f.top; cp.width = width; cp.idx = eidx; cp.n_real = f.E; cp.xin = x; cp.ld_in = width; cp.x = x; cp.ldx = width;
        if (sh) { cp.add = ysh; cp.add_gate = rz + n_out; cp.ld_gate = n_out + 1; }
        np.w = L.norm2; np.eps = info.eps; np.h = h; np.ldh = width;
        EpiParams<AT> eg{}; eg.act = act; eg.lda = f.ff; eg.glu_kind = GLU_SILU;
        EpiParams<AT> ed{}; ed.out = ye; ed.ldo = width; ed.scale = 1.0f;
        if (T == 1) {   // the chosen experts' matrices, picked on the device from the router's list (identity experts have none), the shared one's beside them
            GemvRowsParams<AT, WT> u{};
            u.a = h; u.w = L.wgate; u.w2 = L.wup; u.K = width; u.O = f.ff; u.e = eg; u.bidx = eidx; u.w_bs = (long long)f.ff * width; u.o_bs = f.ff; u.n_mats = f.E;
            if (sh) { u.extra.a = h; u.extra.w = L.sgate; u.extra.w2 = L.sup; u.extra.K = width; u.extra.O = f.shared_ff; u.extra.act = act_sh; }
            if (this->template launch_gemv<EPI_GLU, NORM_NONE>(st, u, f.top + (sh ? 1 : 0))) return 1;
            GemvRowsParams<AT, WT> d{};
            d.a = act; d.w = L.wdown; d.K = f.ff; d.O = width; d.e = ed; d.bidx = eidx; d.a_bs = f.ff; d.w_bs = (long long)width * f.ff; d.o_bs = width; d.n_mats = f.E;
            if (sh) { d.extra.a = act_sh; d.extra.w = L.sdown; d.extra.K = f.shared_ff; d.extra.O = width; d.extra.out = ysh; }
            if (this->template launch_gemv<EPI_STORE, NORM_NONE>(st, d, f.top + (sh ? 1 : 0))) return 1;
            return launch_k("moe_combine_resnorm_kernel", st, pdl_now, moe_combine_resnorm_kernel<AT, true, 4>, dim3(1), dim3(one_row_threads()), 0, np);
        }
        // rows sorted by expert; identity experts sort behind the experts with matrices and take no product
        const int n = T * f.top;
        MoeSortParams sp{};
        sp.idx = eidx; sp.n = n; sp.E = n_out; sp.top = f.top; sp.grp = grp; sp.slot = slot; sp.row_of = row_of;
        if (launch_k("moe_sort_kernel", st, pdl_now, moe_sort_kernel, dim3(1), dim3(1024), (size_t)2 * n_out * 4, sp)) return 1;
        MoeGatherParams<AT> gp{};
        gp.h = h; gp.ld = width; gp.row_of = row_of; gp.out = xg; gp.width = width;
        if (launch_k("moe_gather_kernel", st, pdl_now, moe_gather_kernel<AT>, dim3(n), dim3(128), 0, gp)) return 1;
        if (this->template matmul_grouped<EPI_GLU>(st, n, f.E, grp, T, xg, width, L.wgate, L.wup, width, f.ff, eg)) return 1;
        if (this->template matmul_grouped<EPI_STORE>(st, n, f.E, grp, T, act, f.ff, L.wdown, nullptr, f.ff, width, ed)) return 1;
        cp.slot = slot;
        if (sh) {
            EpiParams<AT> su{}; su.act = act_sh; su.lda = f.shared_ff; su.glu_kind = GLU_SILU;
            if (this->template matmul<EPI_GLU>(st, T, h, width, L.sgate, L.sup, width, f.shared_ff, su)) return 1;
            EpiParams<AT> sd{}; sd.out = ysh; sd.ldo = width; sd.scale = 1.0f;
            if (this->template matmul<EPI_STORE>(st, T, act_sh, f.shared_ff, L.sdown, nullptr, f.shared_ff, width, sd)) return 1;
        }
        if (width <= 8 * 256) return launch_k("moe_combine_resnorm_kernel", st, pdl_now, moe_combine_resnorm_kernel<AT, false, 8>, dim3(T), dim3(256), 0, np);
        return launch_k("moe_combine_resnorm_kernel", st, pdl_now, moe_combine_resnorm_kernel<AT, false, 16>, dim3(T), dim3(256), 0, np);
    }

    int run_layers(cudaStream_t st, int T, const PosSrc& ps, uint32_t pos_hint) override {
        {
            EmbedRowsParams<WT> p{};
            p.embed = embed; p.tokens = d_tokens; p.x = x; p.width = width; p.ps = ps; p.scale = embed_scale; p.h = h;
            embed_rows_kernel<WT><<<T, 128, 0, st>>>(p);
            if (check_launch("embed_rows_kernel")) return 1;
        }
        for (size_t li = 0; li < layers.size(); li++) {
            const Layer& L = layers[li];
            if (mixer(st, L, T, ps, pos_hint)) return 1;
            if (L.f.kind == LU_FF_DENSE && ff_dense(st, L, T)) return 1;
            if (L.f.kind == LU_FF_MOE && ff_moe(st, L, T)) return 1;
            if (this->keep_layer(st, li, T)) return 1;
        }
        return 0;
    }
    int head_rows(cudaStream_t st, int m, const uint32_t* rows_dev, float* out) override {
        EpiParams<AT> e{}; e.out = out; e.ldo = vocab; e.scale = 1.0f;
        if (m == 1 && rows_dev == nullptr) {
            GemvRowsParams<AT, WT> p{};
            p.x = x; p.nw = final_norm; p.eps = info.eps; p.w = embed; p.K = width; p.O = vocab; p.e = e;
            return this->template launch_gemv<EPI_STORE, NORM_RMS>(st, p);
        }
        NormRowsParams<AT> np{};
        np.x = x; np.ldx = width; np.rows = rows_dev; np.w = final_norm; np.out = hn; np.ldo = width; np.n = width; np.eps = info.eps;
        if (launch_k("rmsnorm_rows_kernel", st, pdl_now, rmsnorm_rows_kernel<AT>, dim3(m), dim3(256), 0, np)) return 1;
        return this->template matmul<EPI_STORE>(st, m, hn, width, embed, nullptr, width, vocab, e);
    }

    void set_model_option(const char* name, int value) override {
        if (!strcmp(name, "latent_expand_rows")) this->latent_expand_rows = std::max(2, value);
    }
    // test access: the latent and the rotated key part (as "k" and "v")
    int read_kv(cudaStream_t st, uint32_t layer, uint32_t pos0, uint32_t n, float* k_out, float* v_out) override {
        if (layer >= layers.size() || (size_t)pos0 + n > max_tokens) { error = "read_kv: out of range"; return 1; }
        return this->read_latent(st, layers[layer].mix, pos0, n, k_out, v_out);
    }
};

ArchModel* lutesun_factory(const std::string& dir, const Json& cfg, const ArchOptions& opt, std::string& err) {
    ArchModel* m = nullptr;
    int rc;
    if (opt.dtype == ARCH_F32) {
        auto* g = new LutesunModel<float, float>();
        rc = g->load(dir, cfg, opt);
        m = g;
    } else {
        auto* g = new LutesunModel<__nv_bfloat16, __nv_bfloat16>();
        rc = g->load(dir, cfg, opt);
        m = g;
    }
    if (rc) { err = m->error; delete m; return nullptr; }
    return m;
}

}  // namespace

void register_lutesun() { arch_register("Lutesun", lutesun_factory); }

}  // namespace lmrs
