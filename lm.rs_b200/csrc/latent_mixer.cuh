// latent_mixer.cuh -- attention whose keys and values are up-projections of one cached latent per token plus one rotated key part
// shared by all heads, for the folder architectures that have it (between dense_model.cuh and the model class):
//     [c_raw | kr] = W_dkv h;  c = rms(c_raw) w;  k_h = [W_uk c | rot(kr)],  v_h = W_uv c;   softmax(scale q.k), causal
// with, as configured: queries straight from h (rq == 0) or through a normed latent of their own; rotation of neighbouring pairs or
// of halves; a sliding window; one sigmoid output gate per head from h.
// Short steps run in the latent space: the keys' up-projection is multiplied into the query, the attention kernel sees one shared
// key/value head of size kv_rank (+ rot_dim), and the values' up-projection follows it.  Long portions up-project the cached latents
// they can see to per-head keys and values first (tensor cores) and run ordinary multi-head attention over them.
#pragma once
#include "dense_model.cuh"
#include "mixer_ops.cuh"

namespace lmrs {

struct LatentCfg {
    int H = 0, dn = 0, dr = 0, dv = 0, rk = 0, rq = 0;   // heads; unrotated, rotated and value size of a head; latent sizes (rq 0: none)
    float scale = 1.0f;
    int window = 0;                // 0: all earlier keys
    bool gate = false;             // per-head output gates
    bool halves = false;           // rotation pairs (i, i + rot_dims/2) instead of (2i, 2i+1)
    int rot_dims = 0;
    std::vector<double> rot_f;     // rot_dims / 2 frequencies
    double rot_mult = 1.0;         // of cos and sin
    std::string rot_key;           // equal keys share tables
    bool latent_space_ok = true, per_head_ok = true;
};

template <typename AT, typename WT> class LatentModel : public DenseModel<AT, WT> {
  public:
    typedef DenseModel<AT, WT> D;
    using D::error; using D::dalloc; using D::dfree; using D::need; using D::load_vec; using D::load_stack; using D::launch_k; using D::pdl_now;
    using D::max_tokens; using D::width; using D::info; using D::MAX_SPLIT;

    struct Latent {
        LatentCfg c;
        WT* w_in = nullptr; int in_rows = 0;      // [query or query latent | key/value latent | rotated part | gates] stacked
        float *dq_norm = nullptr, *dkv_norm = nullptr;
        float* cache = nullptr;                   // [max_tokens][rk + dr]
        AT* cache_op = nullptr;                   // [max_tokens][rk] the latent in the operand type
        WT *wuq = nullptr, *wuk = nullptr, *wukT = nullptr, *wuv = nullptr;   // wukT: [H][rk][dn], wuk transposed per head
        Rotation rot{};
    };
    int latent_expand_rows = 16;   // portions of at least this many rows take the per-head form

    // sizes and mask from a mixer entry; rotation frequencies are the architecture's business
    int parse_latent(const Json& m, const std::string& where, LatentCfg& c) {
        c.H = (int)m.at("heads").number(0); c.dn = (int)m.at("dim").number(0); c.dv = (int)m.at("vdim").number(c.dn);
        c.dr = (int)m.at("rot_dim").number(0); c.rk = (int)m.at("kv_rank").number(0);
        c.scale = (float)m.at("scale").number(1.0);
        c.window = m.has("mask") && m.at("mask").is_obj() ? (int)m.at("mask").at("size").number(0) : 0;
        c.rot_dims = m.has("rot") && m.at("rot").is_obj() ? (int)m.at("rot").at("dims").number(c.dr) : 0;
        if (c.H <= 0 || c.dn <= 0 || c.dv <= 0) { error = where + ": bad head geometry"; return 1; }
        if (c.dr < 0 || c.rk <= 0) { error = where + ": rot_dim and kv_rank are required"; return 1; }
        if (c.window < 0) { error = where + ": mask.size must not be negative"; return 1; }
        if (c.rot_dims < 0 || c.rot_dims > c.dr || c.rot_dims % 2 != 0) { error = where + ": rot.dims must be even and at most rot_dim"; return 1; }
        // a latent too wide for the attention kernel's tiles is always up-projected to per-head keys and values
        c.latent_space_ok = D::attention_fits(c.rk + c.dr, c.rk, true);
        c.per_head_ok = D::attention_fits(c.dn + c.dr, c.dv);
        if (!c.latent_space_ok && !c.per_head_ok) { error = where + ": neither kv_rank " + std::to_string(c.rk) + " nor the per-head sizes fit the attention kernel's shared-memory tiles"; return 1; }
        return 0;
    }

    // `q`: prefix of the mixer's tensor names
    int load_latent(const SafeTensors& st, const std::string& q, Latent& L) {
        const LatentCfg& c = L.c;
        const int dq = c.dn + c.dr;
        std::vector<std::pair<std::string, int>> in;
        if (c.rq > 0) in.push_back({q + "dq", c.rq});
        else in.push_back({q + "q", c.H * dq});
        in.push_back({q + "dkv", c.rk + c.dr});
        if (c.gate) in.push_back({q + "g", c.H});
        if (load_stack(st, in, width, &L.w_in, &L.in_rows) || load_vec(st, q + "dkv.norm", c.rk, &L.dkv_norm)) return 1;
        if (c.rq > 0 && (load_vec(st, q + "dq.norm", c.rq, &L.dq_norm) || load_stack(st, {{q + "uq", c.H * dq}}, c.rq, &L.wuq, nullptr))) return 1;
        if (load_stack(st, {{q + "uv", c.H * c.dv}}, c.rk, &L.wuv, nullptr) || load_stack(st, {{q + "uk", c.H * c.dn}}, c.rk, &L.wuk, nullptr)) return 1;
        const StTensor* t = nullptr;
        if (need(st, q + "uk", {c.H * c.dn, c.rk}, &t)) return 1;
        std::vector<float> tr((size_t)c.H * c.rk * c.dn);   // [h][r][d] <- uk[h*dn + d][r]
        for (int hh = 0; hh < c.H; hh++)
            for (int d = 0; d < c.dn; d++)
                for (int r = 0; r < c.rk; r++) {
                    const size_t src = ((size_t)hh * c.dn + d) * c.rk + r;
                    tr[((size_t)hh * c.rk + r) * c.dn + d] =
                        t->dtype == "BF16" ? bf16_bits_to_f32(reinterpret_cast<const uint16_t*>(t->data)[src]) : reinterpret_cast<const float*>(t->data)[src];
                }
        if (dalloc(&L.wukT, tr.size()) || this->upload_host(tr, L.wukT)) return 1;
        if (dalloc(&L.cache, (size_t)max_tokens * (c.rk + c.dr)) || dalloc(&L.cache_op, (size_t)max_tokens * c.rk)) return 1;
        L.rot.dims = c.rot_dims; L.rot.halves = c.halves;
        if (c.rot_dims > 0 && this->angle_tables(c.rot_key, c.rot_f, c.rot_mult, &L.rot.cos, &L.rot.sin)) return 1;
        max_cq = std::max(max_cq, c.rq); max_qraw = std::max(max_qraw, c.rq > 0 ? c.H * dq : 0); max_qn = std::max(max_qn, c.H * c.dn);
        max_q = std::max(max_q, c.H * (std::max(c.rk, c.dn) + c.dr)); max_lat_att = std::max(max_lat_att, c.H * c.rk);
        max_out = std::max(max_out, c.H * c.dv); max_heads = std::max(max_heads, c.H); max_part = std::max(max_part, c.H * (std::max(c.rk, c.dv) + 2));
        max_kfull = std::max(max_kfull, c.H * dq); max_vfull = std::max(max_vfull, c.H * c.dv); max_knope = std::max(max_knope, c.H * c.dn);
        return 0;
    }

    // scratch of the mixer for `rows` rows (nothing when no layer has one)
    int ensure_latent_scratch(size_t rows) {
        for (void* p : {(void*)l_cq, (void*)l_qn, (void*)l_att, (void*)l_out, (void*)l_qraw, (void*)l_q, (void*)l_gate, (void*)l_part}) dfree(p);
        l_cq = l_qn = l_att = l_out = nullptr;
        l_qraw = l_q = l_gate = l_part = nullptr;
        if (max_heads == 0) return 0;
        return dalloc(&l_cq, rows * max_cq) || dalloc(&l_qn, rows * max_qn) || dalloc(&l_att, rows * max_lat_att) || dalloc(&l_out, rows * max_out) ||
               dalloc(&l_qraw, rows * max_qraw) || dalloc(&l_q, rows * max_q) || dalloc(&l_gate, rows * max_heads) || dalloc(&l_part, (size_t)MAX_SPLIT * max_part);
    }

    // from the projected rows `proj` [T][L.in_rows] to the concatenated heads *out [T][H * dv]
    int mixer_latent(cudaStream_t st, const Latent& L, int T, const PosSrc& ps, uint32_t pos_hint, const float* proj, const AT** out) {
        const LatentCfg& c = L.c;
        const int dq = c.dn + c.dr, dl = c.rk + c.dr;
        *out = l_out;
        LatentKvPostParams<AT> kp{};
        kp.in = proj; kp.ld = L.in_rows; kp.rq = c.rq; kp.kv_off = c.rq > 0 ? c.rq : c.H * dq; kp.rk = c.rk; kp.dr = c.dr; kp.wq = L.dq_norm; kp.wkv = L.dkv_norm;
        kp.eps = info.eps; kp.rot = L.rot; kp.cq_out = l_cq; kp.cache = L.cache; kp.cache_op = L.cache_op; kp.ps = ps;
        if (c.gate) { kp.gate_out = l_gate; kp.H = c.H; kp.gate_off = kp.kv_off + dl; }
        if (launch_k("latent_kv_post_kernel", st, pdl_now, latent_kv_post_kernel<AT>, dim3(T), dim3(256), 0, kp)) return 1;
        if (c.rq > 0) {
            EpiParams<AT> eq{}; eq.out = l_qraw; eq.ldo = c.H * dq; eq.scale = 1.0f;
            if (this->template matmul<EPI_STORE>(st, T, l_cq, c.rq, L.wuq, nullptr, c.rq, c.H * dq, eq)) return 1;
        }
        LatentQPostParams<AT> qp{};
        qp.q = c.rq > 0 ? l_qraw : proj; qp.ldq = c.rq > 0 ? c.H * dq : L.in_rows;
        qp.H = c.H; qp.dn = c.dn; qp.dr = c.dr; qp.rk = c.rk; qp.rot = L.rot; qp.qn_out = l_qn; qp.qabs = l_q; qp.ps = ps;
        AttnRowsParams<AT> p{};
        p.q = l_q; p.T = T; p.H = c.H; p.scale = c.scale; p.ps = ps; p.window = c.window; p.gate = c.gate ? l_gate : nullptr;
        if (c.per_head_ok && (!c.latent_space_ok || (T >= latent_expand_rows && !ps.sp))) {
            // per-head form: keys and values of the positions the step can see, j0 .. n, up-projected from the cached latents, then
            // plain attention.  A graph-replayed step does not know its position on the host: it up-projects what any position of its
            // 64-position bucket may see (rows beyond the position are never read by the attention)
            int first = (int)ps.pos, n = (int)ps.pos + T;
            if (ps.sp) {
                const bool bounded = pos_hint / ATT_KT + 1 < (uint32_t)MAX_SPLIT;
                first = bounded ? (int)(pos_hint / ATT_KT * ATT_KT) : -1;
                n = bounded ? (int)std::min<uint32_t>(max_tokens, (pos_hint / ATT_KT + 1) * ATT_KT) : (int)max_tokens;
            }
            const int j0 = c.window > 0 && first >= c.window ? (first - c.window + 1) / ATT_KT * ATT_KT : 0;   // the attention walks whole key tiles
            if (!kfull && (dalloc(&kfull, (size_t)max_tokens * max_kfull) || dalloc(&vfull, (size_t)max_tokens * max_vfull) || dalloc(&knope, (size_t)max_tokens * max_knope)))
                return 1;
            qp.qfull = l_q;
            if (launch_k("latent_q_post_kernel", st, pdl_now, latent_q_post_kernel<AT>, dim3(T, (c.H + 3) / 4), dim3(128), 0, qp)) return 1;
            const AT* lat = L.cache_op + (size_t)j0 * c.rk;
            EpiParams<AT> ek{}; ek.out = knope + (size_t)j0 * c.H * c.dn; ek.ldo = c.H * c.dn; ek.scale = 1.0f;
            if (this->template matmul<EPI_STORE>(st, n - j0, lat, c.rk, L.wuk, nullptr, c.rk, c.H * c.dn, ek)) return 1;
            EpiParams<AT> ev{}; ev.out = vfull + (size_t)j0 * c.H * c.dv; ev.ldo = c.H * c.dv; ev.scale = 1.0f;
            if (this->template matmul<EPI_STORE>(st, n - j0, lat, c.rk, L.wuv, nullptr, c.rk, c.H * c.dv, ev)) return 1;
            LatentExpandParams xp{};
            xp.knope = knope; xp.cache = L.cache; xp.kfull = kfull; xp.H = c.H; xp.dn = c.dn; xp.dr = c.dr; xp.rk = c.rk; xp.j0 = j0;
            if (launch_k("latent_expand_kernel", st, pdl_now, latent_expand_kernel, dim3(n - j0), dim3(256), 0, xp)) return 1;
            p.kcache = kfull; p.vcache = vfull; p.out = l_out; p.G = c.H; p.dk = dq; p.dv = c.dv; p.k_ld = c.H * dq; p.v_ld = c.H * c.dv;
            return this->attention_launch(st, p, l_part, pos_hint);
        }
        if (launch_k("latent_q_post_kernel", st, pdl_now, latent_q_post_kernel<AT>, dim3(T, (c.H + 3) / 4), dim3(128), 0, qp)) return 1;
        // the unrotated query part of head z into the latent space: q[:, z*dl .. z*dl+rk] = qn[:, z*dn ..] . wukT[z]^T
        EpiParams<AT> ea{}; ea.out = l_q; ea.ldo = c.H * dl; ea.scale = 1.0f;
        if (this->template matmul_batched<EPI_STORE>(st, T, c.H, l_qn, c.H * c.dn, c.dn, L.wukT, (long long)c.rk * c.dn, c.dn, c.rk, ea, dl)) return 1;
        // one shared key/value head: keys [latent | rotated part], values = the latent
        p.kcache = L.cache; p.vcache = L.cache; p.out = l_att; p.G = 1; p.dk = dl; p.dv = c.rk; p.k_ld = dl; p.v_ld = dl; p.v_in_k = 1;
        if (this->attention_launch(st, p, l_part, pos_hint)) return 1;
        // values' up-projection per head: out[:, z*dv ..] = att[:, z*rk ..] . wuv[z]^T
        EpiParams<AT> ev{}; ev.act = l_out; ev.lda = c.H * c.dv;
        return this->template matmul_batched<EPI_ACT>(st, T, c.H, l_att, c.H * c.rk, c.rk, L.wuv, (long long)c.dv * c.rk, c.rk, c.dv, ev, c.dv);
    }

    // test access: the cached latents (as "k") and rotated key parts (as "v")
    int read_latent(cudaStream_t st, const Latent& L, uint32_t pos0, uint32_t n, float* k_out, float* v_out) {
        const size_t dl = (size_t)L.c.rk + L.c.dr;
        GCK(cudaStreamSynchronize(st));
        GCK(cudaMemcpy2D(k_out, (size_t)L.c.rk * 4, L.cache + pos0 * dl, dl * 4, (size_t)L.c.rk * 4, n, cudaMemcpyDeviceToHost));
        if (L.c.dr > 0) GCK(cudaMemcpy2D(v_out, (size_t)L.c.dr * 4, L.cache + pos0 * dl + L.c.rk, dl * 4, (size_t)L.c.dr * 4, n, cudaMemcpyDeviceToHost));
        return 0;
    }

  private:
    AT *l_cq = nullptr, *l_qn = nullptr, *l_att = nullptr, *l_out = nullptr;
    float *l_qraw = nullptr, *l_q = nullptr, *l_gate = nullptr, *l_part = nullptr;
    float *kfull = nullptr, *vfull = nullptr, *knope = nullptr;   // per-head keys and values of all cached positions (per-head form)
    int max_cq = 0, max_qraw = 0, max_qn = 0, max_q = 0, max_lat_att = 0, max_out = 0, max_heads = 0, max_part = 0, max_kfull = 0, max_vfull = 0, max_knope = 0;
};

}  // namespace lmrs
