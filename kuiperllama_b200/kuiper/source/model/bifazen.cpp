#include "model/bifazen.h"

#include <cmath>
#include <string>
#include <vector>

namespace model {
KLLM_REGISTER_SEQUENCE_MODEL("Bifazen", BifazenModel);

namespace {
int32_t get_int(const json::Value& v, const char* key) { return static_cast<int32_t>(v.at(key).as_int()); }
double get_number(const json::Value& v, const char* key) { return v.at(key).as_number(); }
bool present(const json::Value& v, const char* key) { return v.has(key) && !v.at(key).is_null(); }
bool shaped(const StTensor* t, int64_t rows, int64_t cols) {
  return t != nullptr && t->shape.size() == 2 && t->shape[0] == rows && t->shape[1] == cols;
}
bool sized(const StTensor* t, int64_t n) { return t != nullptr && t->shape.size() == 1 && t->shape[0] == n; }
base::Status bad(const std::string& p, const char* what) { return base::error::ModelParseError(p + ": " + what); }
bool blends(const json::Value& mixer) { return present(mixer, "v_mix") && mixer.at("v_mix").as_bool(); }
int32_t window_of(const json::Value& mixer) { return present(mixer, "mask") ? get_int(mixer.at("mask"), "size") : 0; }
}  // namespace

base::Status BifazenModel::centred_norm(const SafetensorsFile& w, const std::string& name, kllm_seq_norm* out) {
  base::Status st;
  std::vector<float> g;
  if (st = read_values(need(w, name, &st), width_, &g); !st) return st;
  for (float& v : g) v += 1.0f;
  out->b = nullptr, out->kind = KLLM_SEQ_NORM_RMS;
  return upload_values(g, &out->w);
}

base::Status BifazenModel::hyper(const SafetensorsFile& w, const std::string& p, kllm_seq_hyper* out) {
  base::Status st;
  const StTensor *in = need(w, p + "in", &st), *o = need(w, p + "out", &st), *mix = need(w, p + "mix", &st);
  if (!st) return st;
  if (!sized(in, streams_) || !sized(o, streams_) || !shaped(mix, streams_, streams_))
    return bad(p, "tensor shapes do not fit the number of streams");
  if (st = upload_f32(in, streams_, &out->in); !st) return st;
  if (st = upload_f32(o, streams_, &out->out); !st) return st;
  return upload_f32(mix, int64_t(streams_) * streams_, &out->mix);
}

base::Status BifazenModel::build_latent(const json::Value& c, const SafetensorsFile& w, const std::string& p, kllm_seq_latent* a) {
  a->heads = get_int(c, "heads"), a->dim = get_int(c, "dim"), a->rot_dim = get_int(c, "rot_dim"), a->vdim = get_int(c, "vdim");
  a->kv_rank = get_int(c, "kv_rank"), a->q_rank = 0;  // the queries have no latent of their own
  a->scale = static_cast<float>(get_number(c, "scale"));
  a->window = window_of(c);
  a->gate = KLLM_SEQ_GATE_NONE, a->sink = nullptr;
  a->rope_dims = 0, a->rope_base = 1.f, a->rope_pairing = KLLM_SEQ_ROPE_PAIRS, a->rope_freq = nullptr;
  if (a->heads <= 0 || a->dim <= 0 || a->rot_dim < 0 || a->vdim <= 0 || a->kv_rank <= 0 || a->window < 0)
    return bad(p, "bad mixer configuration");
  base::Status st;
  if (present(c, "rot")) {
    a->rope_dims = get_int(c.at("rot"), "dims");
    const double base = get_number(c.at("rot"), "base");
    if (a->rope_dims < 0 || a->rope_dims > a->rot_dim || (a->rope_dims & 1) || !(base > 0.0))
      return bad(p, "bad rotary configuration");
    a->rope_base = static_cast<float>(base);
    std::vector<float> freq(static_cast<size_t>(a->rope_dims / 2));
    for (size_t i = 0; i < freq.size(); ++i)
      freq[i] = static_cast<float>(std::pow(base, -2.0 * static_cast<double>(i) / a->rope_dims));
    if (!freq.empty())
      if (st = upload_values(freq, &a->rope_freq); !st) return st;
  }
  const StTensor *q = need(w, p + "q", &st), *dkv = need(w, p + "dkv", &st), *norm = need(w, p + "dkv.norm", &st),
                 *uk = need(w, p + "uk", &st), *uv = need(w, p + "uv", &st), *o = need(w, p + "o", &st);
  if (!st) return st;
  const int64_t H = a->heads;
  if (!shaped(q, H * (a->dim + a->rot_dim), width_) || !shaped(dkv, a->kv_rank + a->rot_dim, width_) ||
      !sized(norm, a->kv_rank) || !shaped(uk, H * a->dim, a->kv_rank) || !shaped(uv, H * a->vdim, a->kv_rank) ||
      !shaped(o, width_, H * a->vdim))
    return bad(p, "tensor shapes do not fit the configuration");
  if (st = upload_compute({q, dkv}, width_, &a->w_in); !st) return st;
  // one tensor holds both expansions, so that a prompt runs them as one product
  if (st = upload_compute({uk, uv}, a->kv_rank, &a->w_uk); !st) return st;
  const size_t es = compute_ == ComputeType::kBFloat16 ? 2 : 4;
  a->w_uv = static_cast<const char*>(a->w_uk) + static_cast<size_t>(H * a->dim) * a->kv_rank * es;
  if (st = upload_compute({o}, H * a->vdim, &a->w_out); !st) return st;
  return upload_f32(norm, a->kv_rank, &a->kv_norm_w);
}

base::Status BifazenModel::build_attention(const json::Value& c, const SafetensorsFile& w, const std::string& p, int32_t v_blend,
                                           kllm_seq_attention* a) {
  a->heads = get_int(c, "heads"), a->kv_heads = get_int(c, "kv_heads"), a->dim = get_int(c, "dim"), a->vdim = get_int(c, "vdim");
  a->scale = static_cast<float>(get_number(c, "scale"));
  a->window = window_of(c);
  if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 || a->window < 0)
    return bad(p, "bad mixer configuration");
  a->gate = KLLM_SEQ_GATE_HEAD, a->qk_norm = KLLM_SEQ_QKNORM_PROJECTION, a->rope_dims = 0, a->v_blend = v_blend;
  const int64_t qn = int64_t(a->heads) * a->dim, kn = int64_t(a->kv_heads) * a->dim, vn = int64_t(a->kv_heads) * a->vdim;
  const int64_t on = int64_t(a->heads) * a->vdim;
  base::Status st;
  const StTensor *q = need(w, p + "q", &st), *k = need(w, p + "k", &st), *v = need(w, p + "v", &st), *g = need(w, p + "g", &st),
                 *o = need(w, p + "o", &st), *qb = need(w, p + "q.b", &st), *kb = need(w, p + "k.b", &st),
                 *vb = need(w, p + "v.b", &st), *ob = need(w, p + "o.b", &st), *qnorm = need(w, p + "q.norm", &st),
                 *knorm = need(w, p + "k.norm", &st);
  if (!st) return st;
  if (!shaped(q, qn, width_) || !shaped(k, kn, width_) || !shaped(v, vn, width_) || !shaped(g, a->heads, width_) ||
      !shaped(o, width_, on) || !sized(qb, qn) || !sized(kb, kn) || !sized(vb, vn) || !sized(ob, width_) || !sized(qnorm, qn) ||
      !sized(knorm, kn))
    return bad(p, "tensor shapes do not fit the configuration");
  if (st = upload_compute({q, k, v, g}, width_, &a->w_in); !st) return st;
  if (st = upload_compute({o}, on, &a->w_out); !st) return st;
  // one bias for the stacked projection; the gate rows have none
  std::vector<float> bias, one;
  const StTensor* parts[] = {qb, kb, vb};
  const int64_t numel[] = {qn, kn, vn};
  for (int i = 0; i < 3; ++i) {
    if (st = read_values(parts[i], numel[i], &one); !st) return st;
    bias.insert(bias.end(), one.begin(), one.end());
  }
  bias.resize(bias.size() + static_cast<size_t>(a->heads), 0.f);
  if (st = upload_values(bias, &a->in_bias); !st) return st;
  if (st = upload_f32(ob, width_, &a->out_bias); !st) return st;
  if (st = upload_f32(qnorm, qn, &a->q_norm_w); !st) return st;
  if (st = upload_f32(knorm, kn, &a->k_norm_w); !st) return st;
  if (v_blend == KLLM_SEQ_VBLEND_MIX) {
    if (st = read_values(need(w, p + "vmix", &st), 1, &one); !st) return st;
    a->v_lambda = one[0];
  }
  return base::error::Success();
}

base::Status BifazenModel::build_dense(const json::Value& c, const SafetensorsFile& w, const std::string& p, kllm_seq_dense* f) {
  f->ff = get_int(c, "ff");
  if (f->ff <= 0) return bad(p, "bad size");
  base::Status st;
  const StTensor *gate = need(w, p + "gate", &st), *up = need(w, p + "up", &st), *down = need(w, p + "down", &st);
  if (!st) return st;
  if (!shaped(gate, f->ff, width_) || !shaped(up, f->ff, width_) || !shaped(down, width_, f->ff))
    return bad(p, "tensor shapes do not fit the configuration");
  f->act = KLLM_SEQ_ACT_GELU_GATE, f->act_a = 0.f, f->act_b = 0.f;
  if (st = upload_compute({gate, up}, width_, &f->up); !st) return st;
  return upload_compute({down}, f->ff, &f->down);
}

// every tensor the configuration implies, by name
base::Status BifazenModel::check_folder(const json::Value& config, const SafetensorsFile& w) {
  base::Status st;
  for (const char* name : {"embed", "final.norm"}) need(w, name, &st);
  const auto& layers = config.at("layers").array;
  bool source = false;
  for (size_t i = 0; i < layers.size(); ++i) {
    const std::string p = "l" + std::to_string(i) + ".";
    const std::string& type = layers[i].at("type").as_string();
    std::vector<std::string> names = {"norm1"};
    if (type == "latent_attention") {
      for (const char* n : {"q", "dkv", "dkv.norm", "uk", "uv", "o"}) names.push_back(std::string("mix.") + n);
    } else if (type == "attention") {
      for (const char* n : {"q", "q.b", "q.norm", "k", "k.b", "k.norm", "v", "v.b", "g", "o", "o.b"})
        names.push_back(std::string("mix.") + n);
      if (blends(layers[i].at("mixer"))) {
        if (source) names.push_back("mix.vmix");
        source = true;
      }
    } else {
      return base::error::FunctionNotImplement("layer " + std::to_string(i) + ": unknown mixer '" + type + "'");
    }
    const bool ff = present(layers[i], "mlp");
    if (ff) {
      const std::string& kind = layers[i].at("mlp").at("kind").as_string();
      if (kind != "dense")
        return base::error::FunctionNotImplement("layer " + std::to_string(i) + ": unknown feed-forward '" + kind + "'");
      for (const char* n : {"norm2", "mlp.gate", "mlp.up", "mlp.down"}) names.push_back(n);
    }
    if (present(config, "streams"))
      for (const char* hc : {"hc1.", "hc2."})
        if (ff || hc[2] == '1')
          for (const char* n : {"in", "out", "mix"}) names.push_back(std::string(hc) + n);
    for (const std::string& n : names) need(w, p + n, &st);
  }
  return st;
}

base::Status BifazenModel::build(const json::Value& config, const SafetensorsFile& w) {
  vocab_ = get_int(config, "vocab");
  width_ = get_int(config, "width");
  norm_eps_ = static_cast<float>(get_number(config.at("norm"), "eps"));
  streams_ = present(config, "streams") ? get_int(config, "streams") : 0;  // absent: one plain residual
  if (vocab_ <= 0 || width_ <= 0) return base::error::ModelParseError("bad vocab / width");
  if (present(config, "streams") && streams_ <= 0) return base::error::ModelParseError("bad number of streams");
  const auto& layers = config.at("layers").array;
  if (layers.empty()) return base::error::ModelParseError("no layers");
  base::Status st;
  layers_.assign(layers.size(), kllm_seq_layer{});
  run_layer_.clear(), run_add_.clear(), run_embed_.clear();
  bool source = false;  // has a layer whose values the later ones blend with been seen?
  for (size_t i = 0; i < layers.size(); ++i) {
    const json::Value& lc = layers[i];
    kllm_seq_layer& L = layers_[i];
    const std::string p = "l" + std::to_string(i) + ".";
    const std::string& type = lc.at("type").as_string();
    const json::Value& mc = lc.at("mixer");
    if (st = centred_norm(w, p + "norm1", &L.pre_mixer); !st) return st;
    if (streams_ > 0)
      if (st = hyper(w, p + "hc1.", &L.hyper_mixer); !st) return st;
    if (type == "latent_attention") {
      L.mixer_kind = KLLM_SEQ_MIXER_LATENT;
      if (st = build_latent(mc, w, p + "mix.", &L.latent); !st) return st;
    } else if (type == "attention") {
      L.mixer_kind = KLLM_SEQ_MIXER_ATTENTION;
      int32_t blend = KLLM_SEQ_VBLEND_NONE;
      if (blends(mc)) {
        blend = source ? KLLM_SEQ_VBLEND_MIX : KLLM_SEQ_VBLEND_SOURCE;
        source = true;
      }
      if (st = build_attention(mc, w, p + "mix.", blend, &L.attn); !st) return st;
    } else {
      return base::error::FunctionNotImplement("layer " + std::to_string(i) + ": unknown mixer '" + type + "'");
    }
    L.ff_kind = KLLM_SEQ_FF_NONE;
    if (present(lc, "mlp")) {
      const json::Value& fc = lc.at("mlp");
      const std::string& kind = fc.at("kind").as_string();
      if (kind != "dense")
        return base::error::FunctionNotImplement("layer " + std::to_string(i) + ": unknown feed-forward '" + kind + "'");
      L.ff_kind = KLLM_SEQ_FF_DENSE;
      if (st = build_dense(fc, w, p + "mlp.", &L.dense); !st) return st;
      if (st = centred_norm(w, p + "norm2", &L.pre_ff); !st) return st;
      if (streams_ > 0)
        if (st = hyper(w, p + "hc2.", &L.hyper_ff); !st) return st;
    }
    run_layer_.push_back(static_cast<int32_t>(i)), run_add_.push_back(-1), run_embed_.push_back(0);
  }
  const StTensor* embed = need(w, "embed", &st);
  if (!st) return st;
  if (!shaped(embed, vocab_, width_)) return base::error::ModelParseError("embed does not fit vocab x width");
  if (st = upload_compute({embed}, width_, &embed_); !st) return st;
  head_ = embed_;  // the classifier is the embedding table itself
  return centred_norm(w, "final.norm", &final_norm_);
}
}  // namespace model
