#include "model/mobatar.h"

#include <cmath>
#include <string>
#include <vector>

namespace model {
KLLM_REGISTER_SEQUENCE_MODEL("Mobatar", MobatarModel);

namespace {
constexpr float kGateSlope = 1.702f;  // of the feed-forward's sigmoid

int32_t get_int(const json::Value& v, const char* key) { return static_cast<int32_t>(v.at(key).as_int()); }
double get_number(const json::Value& v, const char* key) { return v.at(key).as_number(); }
bool present(const json::Value& v, const char* key) { return v.has(key) && !v.at(key).is_null(); }
bool shaped(const StTensor* t, int64_t rows, int64_t cols) {
  return t != nullptr && t->shape.size() == 2 && t->shape[0] == rows && t->shape[1] == cols;
}
bool sized(const StTensor* t, int64_t n) { return t != nullptr && t->shape.size() == 1 && t->shape[0] == n; }
base::Status bad(const std::string& p, const char* what) { return base::error::ModelParseError(p + ": " + what); }
int32_t mask_of(const json::Value& mixer) { return present(mixer, "mask") ? get_int(mixer.at("mask"), "size") : 0; }

// The angle per position of pair i, base^(-2 i / dims), under a "scaling" entry: a factor alone divides every frequency; with
// "original" a frequency is kept when its wavelength is short against the original context, divided when it is long, and
// blended in between.
std::vector<float> frequencies(const json::Value& rot, int32_t dims, double base) {
  constexpr double kTurn = 6.283185307179586;
  std::vector<float> out(static_cast<size_t>(dims / 2));
  for (size_t i = 0; i < out.size(); ++i) {
    double f = std::pow(base, -2.0 * static_cast<double>(i) / dims);
    if (present(rot, "scaling")) {
      const json::Value& s = rot.at("scaling");
      const double factor = get_number(s, "factor");
      if (!present(s, "original")) {
        f /= factor;
      } else {
        const double original = get_number(s, "original"), low = get_number(s, "low"), high = get_number(s, "high");
        const double wavelength = kTurn / f;
        if (wavelength > original / low) {
          f /= factor;
        } else if (wavelength >= original / high) {
          const double keep = (original / wavelength - low) / (high - low);
          f = (1.0 - keep) * f / factor + keep * f;
        }
      }
    }
    out[i] = static_cast<float>(f);
  }
  return out;
}

// the entry whose tensors entry i uses; negative when the chain leaves the list or never ends
int owner_of(const std::vector<json::Value>& layers, size_t i) {
  for (size_t hops = 0; hops <= layers.size(); ++hops) {
    if (!present(layers[i], "weights_of")) return static_cast<int>(i);
    const int64_t j = layers[i].at("weights_of").as_int();
    if (j < 0 || j >= static_cast<int64_t>(layers.size())) return -1;
    i = static_cast<size_t>(j);
  }
  return -1;
}
}  // namespace

base::Status MobatarModel::centred_norm(const SafetensorsFile& w, const std::string& name, kllm_seq_norm* out) {
  base::Status st;
  std::vector<float> g;
  if (st = read_values(need(w, name, &st), width_, &g); !st) return st;
  for (float& v : g) v += 1.0f;
  out->b = nullptr, out->kind = KLLM_SEQ_NORM_RMS;
  return upload_values(g, &out->w);
}

base::Status MobatarModel::build_rotation(const json::Value& c, const std::string& p, int32_t limit, int32_t* dims, float* base,
                                          const float** freq) {
  *dims = 0, *base = 1.f, *freq = nullptr;
  if (!present(c, "rot")) return base::error::Success();
  const json::Value& rot = c.at("rot");
  *dims = get_int(rot, "dims");
  const double b = get_number(rot, "base");
  if (*dims < 0 || *dims > limit || (*dims & 1) || !(b > 0.0)) return bad(p, "bad rotary configuration");
  *base = static_cast<float>(b);
  return *dims > 0 ? upload_values(frequencies(rot, *dims, b), freq) : base::error::Success();
}

base::Status MobatarModel::build_attention(const json::Value& c, const SafetensorsFile& w, const std::string& p, bool gated,
                                           kllm_seq_attention* a) {
  a->heads = get_int(c, "heads"), a->kv_heads = get_int(c, "kv_heads"), a->dim = get_int(c, "dim"), a->vdim = get_int(c, "vdim");
  a->scale = static_cast<float>(get_number(c, "scale"));
  a->window = 0, a->chunk = mask_of(c);
  if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 || a->chunk < 0)
    return bad(p, "bad mixer configuration");
  base::Status st = build_rotation(c, p, a->dim, &a->rope_dims, &a->rope_base, &a->rope_freq);
  if (!st) return st;
  a->rope_pairing = KLLM_SEQ_ROPE_HALVES;
  a->gate = gated ? KLLM_SEQ_GATE_HEAD : KLLM_SEQ_GATE_NONE;
  a->qk_norm = gated ? KLLM_SEQ_QKNORM_PROJECTION : KLLM_SEQ_QKNORM_UNIT;
  const int64_t qn = int64_t(a->heads) * a->dim, kn = int64_t(a->kv_heads) * a->dim, vn = int64_t(a->kv_heads) * a->vdim;
  const int64_t on = int64_t(a->heads) * a->vdim;
  const StTensor *q = need(w, p + "q", &st), *k = need(w, p + "k", &st), *v = need(w, p + "v", &st), *o = need(w, p + "o", &st);
  if (!st) return st;
  if (!shaped(q, qn, width_) || !shaped(k, kn, width_) || !shaped(v, vn, width_) || !shaped(o, width_, on))
    return bad(p, "tensor shapes do not fit the configuration");
  if (st = upload_compute({o}, on, &a->w_out); !st) return st;
  if (!gated) {
    // the one in the denominator is a sink whose score is 0
    if (st = upload_values(std::vector<float>(static_cast<size_t>(a->heads), 0.f), &a->sink); !st) return st;
    return upload_compute({q, k, v}, width_, &a->w_in);
  }
  const StTensor *g = need(w, p + "g", &st), *qnorm = need(w, p + "q.norm", &st), *knorm = need(w, p + "k.norm", &st);
  if (!st) return st;
  if (!shaped(g, a->heads, width_) || !sized(qnorm, qn) || !sized(knorm, kn))
    return bad(p, "tensor shapes do not fit the configuration");
  if (st = upload_f32(qnorm, qn, &a->q_norm_w); !st) return st;
  if (st = upload_f32(knorm, kn, &a->k_norm_w); !st) return st;
  return base::error::Success();  // the input projection is stacked with the other mixer's
}

base::Status MobatarModel::build_retention(const json::Value& c, const SafetensorsFile& w, const std::string& p,
                                           kllm_seq_linear* a) {
  a->heads = get_int(c, "heads"), a->dim = get_int(c, "dim"), a->vdim = get_int(c, "vdim");
  if (a->heads <= 0 || a->dim <= 0 || a->vdim <= 0) return bad(p, "bad mixer configuration");
  base::Status st = build_rotation(c, p, a->dim, &a->rope_dims, &a->rope_base, &a->rope_freq);
  if (!st) return st;
  a->rope_pairing = KLLM_SEQ_ROPE_HALVES;
  a->qkv_act = KLLM_SEQ_QKV_PLAIN, a->out_norm = KLLM_SEQ_OUTNORM_HEAD, a->gate_act = KLLM_SEQ_GATEACT_SILU;
  a->k_scale = static_cast<float>(1.0 / std::sqrt(static_cast<double>(a->dim)));
  std::vector<float> decay;
  for (const json::Value& d : c.at("decay").array) decay.push_back(static_cast<float>(d.as_number()));
  if (static_cast<int32_t>(decay.size()) != a->heads) return bad(p, "one decay per head is needed");
  for (float d : decay)
    if (!(d >= 0.f)) return bad(p, "a decay is negative");
  if (st = upload_values(decay, &a->decay); !st) return st;
  const int64_t qn = int64_t(a->heads) * a->dim, vn = int64_t(a->heads) * a->vdim;
  const StTensor *q = need(w, p + "q", &st), *k = need(w, p + "k", &st), *v = need(w, p + "v", &st), *g = need(w, p + "g", &st),
                 *o = need(w, p + "o", &st);
  if (!st) return st;
  if (!shaped(q, qn, width_) || !shaped(k, qn, width_) || !shaped(v, vn, width_) || !shaped(g, vn, width_) ||
      !shaped(o, width_, vn))
    return bad(p, "tensor shapes do not fit the configuration");
  return upload_compute({o}, vn, &a->w_out);  // the input projection is stacked with the other mixer's
}

base::Status MobatarModel::build_latent(const json::Value& c, const SafetensorsFile& w, const std::string& p, kllm_seq_latent* a) {
  a->heads = get_int(c, "heads"), a->dim = get_int(c, "dim"), a->rot_dim = get_int(c, "rot_dim"), a->vdim = get_int(c, "vdim");
  a->kv_rank = get_int(c, "kv_rank"), a->q_rank = 0;  // the queries have no latent of their own
  a->scale = static_cast<float>(get_number(c, "scale"));
  a->window = mask_of(c);
  a->gate = KLLM_SEQ_GATE_NONE, a->sink = nullptr, a->rope_pairing = KLLM_SEQ_ROPE_PAIRS;
  if (a->heads <= 0 || a->dim <= 0 || a->rot_dim < 0 || a->vdim <= 0 || a->kv_rank <= 0 || a->window < 0)
    return bad(p, "bad mixer configuration");
  base::Status st = build_rotation(c, p, a->rot_dim, &a->rope_dims, &a->rope_base, &a->rope_freq);
  if (!st) return st;
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

base::Status MobatarModel::build_dense(const json::Value& c, const SafetensorsFile& w, const std::string& p, kllm_seq_dense* f) {
  f->ff = get_int(c, "ff");
  if (f->ff <= 0) return bad(p, "bad size");
  f->act = KLLM_SEQ_ACT_CLAMP_SWIGLU, f->act_a = static_cast<float>(get_number(c, "limit")), f->act_b = kGateSlope;
  base::Status st;
  const StTensor *gate = need(w, p + "gate", &st), *up = need(w, p + "up", &st), *down = need(w, p + "down", &st),
                 *gb = need(w, p + "gate.b", &st), *ub = need(w, p + "up.b", &st), *db = need(w, p + "down.b", &st);
  if (!st) return st;
  if (!shaped(gate, f->ff, width_) || !shaped(up, f->ff, width_) || !shaped(down, width_, f->ff) || !sized(gb, f->ff) ||
      !sized(ub, f->ff) || !sized(db, width_))
    return bad(p, "tensor shapes do not fit the configuration");
  if (st = upload_compute({gate, up}, width_, &f->up); !st) return st;
  if (st = upload_compute({down}, f->ff, &f->down); !st) return st;
  if (st = upload_f32_parts({gb, ub}, {f->ff, f->ff}, &f->up_bias); !st) return st;
  return upload_f32(db, width_, &f->down_bias);
}

// every tensor the configuration implies, by name
base::Status MobatarModel::check_folder(const json::Value& config, const SafetensorsFile& w) {
  base::Status st;
  for (const char* name : {"embed", "bigram", "final.norm", "head"}) need(w, name, &st);
  const auto& layers = config.at("layers").array;
  for (size_t i = 0; i < layers.size(); ++i) {
    const std::string where = "layer " + std::to_string(i), p = "l" + std::to_string(i) + ".";
    const int own = owner_of(layers, i);
    if (own < 0) return base::error::ModelParseError(where + ": 'weights_of' names no layer");
    if (own != static_cast<int>(i)) continue;
    const std::string& type = layers[i].at("type").as_string();
    std::vector<std::string> names = {"norm1"};
    if (type == "attention") {
      for (const char* n : {"q", "k", "v", "o"}) names.push_back(std::string("mix.") + n);
    } else if (type == "parallel") {
      for (const char* n : {"q", "q.norm", "k", "k.norm", "v", "g", "o"}) names.push_back(std::string("mix.left.") + n);
      for (const char* n : {"q", "k", "v", "g", "o"}) names.push_back(std::string("mix.right.") + n);
    } else if (type == "latent_attention") {
      for (const char* n : {"q", "dkv", "dkv.norm", "uk", "uv", "o"}) names.push_back(std::string("mix.") + n);
    } else {
      return base::error::FunctionNotImplement(where + ": unknown mixer '" + type + "'");
    }
    if (present(layers[i], "mlp")) {
      const std::string& kind = layers[i].at("mlp").at("kind").as_string();
      if (kind != "dense") return base::error::FunctionNotImplement(where + ": unknown feed-forward '" + kind + "'");
      for (const char* n : {"norm2", "mlp.gate", "mlp.gate.b", "mlp.up", "mlp.up.b", "mlp.down", "mlp.down.b"}) names.push_back(n);
    }
    for (const std::string& n : names) need(w, p + n, &st);
  }
  return st;
}

base::Status MobatarModel::build(const json::Value& config, const SafetensorsFile& w) {
  vocab_ = get_int(config, "vocab");
  width_ = get_int(config, "width");
  norm_eps_ = static_cast<float>(get_number(config.at("norm"), "eps"));
  if (vocab_ <= 0 || width_ <= 0) return base::error::ModelParseError("bad vocab / width");
  const auto& layers = config.at("layers").array;
  if (layers.empty()) return base::error::ModelParseError("no layers");
  base::Status st;
  layers_.clear();
  run_layer_.clear(), run_add_.clear(), run_embed_.clear();
  std::vector<int32_t> slot(layers.size(), -1);  // where an entry's own weights are in layers_
  for (size_t i = 0; i < layers.size(); ++i) {
    const json::Value& lc = layers[i];
    const std::string where = "layer " + std::to_string(i);
    const int own = owner_of(layers, i);
    if (own < 0) return base::error::ModelParseError(where + ": 'weights_of' names no layer");
    if (own != static_cast<int>(i)) continue;
    slot[i] = static_cast<int32_t>(layers_.size());
    layers_.push_back(kllm_seq_layer{});
    kllm_seq_layer& L = layers_.back();
    const std::string p = "l" + std::to_string(i) + ".";
    const std::string& type = lc.at("type").as_string();
    const json::Value& mc = lc.at("mixer");
    L.pre_mixer.kind = L.pre_ff.kind = KLLM_SEQ_NORM_NONE;  // the sublayers read x itself
    if (st = centred_norm(w, p + "norm1", &L.post_mixer); !st) return st;
    if (type == "attention") {
      L.mixer_kind = KLLM_SEQ_MIXER_ATTENTION;
      if (st = build_attention(mc, w, p + "mix.", false, &L.attn); !st) return st;
    } else if (type == "parallel") {
      L.mixer_kind = KLLM_SEQ_MIXER_ATTENTION, L.mixer2_kind = KLLM_SEQ_MIXER_LINEAR;
      L.mixer_scale = static_cast<float>(get_number(mc, "left_scale"));
      L.mixer2_scale = static_cast<float>(get_number(mc, "right_scale"));
      if (st = build_attention(mc.at("left"), w, p + "mix.left.", true, &L.attn); !st) return st;
      if (st = build_retention(mc.at("right"), w, p + "mix.right.", &L.linear); !st) return st;
      // one tensor holds both input projections, so that a step runs them as one product
      std::vector<const StTensor*> in;
      for (const char* n : {"left.q", "left.k", "left.v", "left.g", "right.q", "right.k", "right.v", "right.g"})
        in.push_back(need(w, p + "mix." + n, &st));
      if (!st) return st;
      if (st = upload_compute(in, width_, &L.attn.w_in); !st) return st;
      const int64_t left = int64_t(L.attn.heads + L.attn.kv_heads) * L.attn.dim + int64_t(L.attn.kv_heads) * L.attn.vdim + L.attn.heads;
      const size_t es = compute_ == ComputeType::kBFloat16 ? 2 : 4;
      L.linear.w_in = static_cast<const char*>(L.attn.w_in) + static_cast<size_t>(left) * width_ * es;
    } else if (type == "latent_attention") {
      L.mixer_kind = KLLM_SEQ_MIXER_LATENT;
      if (st = build_latent(mc, w, p + "mix.", &L.latent); !st) return st;
    } else {
      return base::error::FunctionNotImplement(where + ": unknown mixer '" + type + "'");
    }
    L.ff_kind = KLLM_SEQ_FF_NONE;
    if (present(lc, "mlp")) {
      const json::Value& fc = lc.at("mlp");
      const std::string& kind = fc.at("kind").as_string();
      if (kind != "dense") return base::error::FunctionNotImplement(where + ": unknown feed-forward '" + kind + "'");
      L.ff_kind = KLLM_SEQ_FF_DENSE;
      if (st = build_dense(fc, w, p + "mlp.", &L.dense); !st) return st;
      if (st = centred_norm(w, p + "norm2", &L.post_ff); !st) return st;
    }
  }
  for (size_t i = 0; i < layers.size(); ++i)
    run_layer_.push_back(slot[static_cast<size_t>(owner_of(layers, i))]), run_add_.push_back(-1), run_embed_.push_back(0);
  const StTensor *embed = need(w, "embed", &st), *bigram = need(w, "bigram", &st), *head = need(w, "head", &st);
  if (!st) return st;
  const json::Value& bc = config.at("embedding").at("bigram");
  bigram_buckets_ = get_int(bc, "buckets");
  bigram_mul_prev_ = bc.at("mul_prev").as_int(), bigram_mul_cur_ = bc.at("mul_cur").as_int();
  if (bigram_buckets_ <= 0 || bigram_mul_prev_ < 0 || bigram_mul_cur_ < 0) return base::error::ModelParseError("bad bigram embedding");
  if (!shaped(embed, vocab_, width_) || !shaped(head, vocab_, width_))
    return base::error::ModelParseError("embed / head do not fit vocab x width");
  if (!shaped(bigram, int64_t(bigram_buckets_) + 1, width_)) return base::error::ModelParseError("bigram does not fit (buckets + 1) x width");
  if (st = upload_compute({embed}, width_, &embed_); !st) return st;
  if (st = upload_compute({bigram}, width_, &bigram_); !st) return st;
  if (st = upload_compute({head}, width_, &head_); !st) return st;
  return centred_norm(w, "final.norm", &final_norm_);
}
}  // namespace model
