"""Nidorax laid out as a ModelSpec: a decoder whose config lists its layers one by one and whose norms stand behind the
residual sums.

Every sublayer reads the residual stream itself and its output joins it inside a norm: x <- norm(alpha x + sublayer(x)), an
RMS norm whose weight is stored around zero.  The mixer is
  lightning         a recurrence over a matrix state per head with one fixed decay per head, on silu projections; one RMS norm
                    over all heads together, a sigmoid gate;
  latent_attention  queries straight from x, keys and values from one cached latent per token plus one rotated key part shared
                    by the heads (rotate-half with YaRN frequencies); a layer may read the latents an earlier layer cached.
The feed-forward is a mixture of squared-relu experts (softmax scores over all experts, a correction that enters the choice
only, the best groups of experts, weights renormalised), or absent.  The logits pass the same norm and the embedding table.
Tensors: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`.
"""
from __future__ import annotations

from ..config.model_config import NidoraxConfig, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec

WEIGHT_SUM_EPS = 1e-20      # added to the chosen experts' sum of scores before they are divided by it


def _mixer(cfg: NidoraxConfig, kind: str, m: dict, prefix: str) -> PartSpec:
    W, eps = cfg.width, cfg.norm_eps
    if kind == "lightning":
        return PartSpec("lightning", {"hidden_size": W, "num_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
                                      "decay": m["decay"], "eps": eps}, prefix)
    position = PartSpec("rope_pairs", {"dims": m["rot_dims"], "base": m["rot_base"], "layout": "halves", "scaling": m["rot_scaling"],
                                       "scaling_kind": "yarn"}) if m["rot_dims"] else None
    return PartSpec("latent_attention", {
        "hidden_size": W, "num_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"], "rank": m["kv_rank"],
        "scale": m["scale"], "eps": eps, "gated": False, "rot_dim": m["rot_dim"], "position": position,
        "shares_cache": m["kv_from"] is not None}, prefix)


def build_nidorax_spec(cfg: NidoraxConfig) -> ModelSpec:
    W = cfg.width
    norm = lambda prefix: PartSpec("rmsnorm", {"size": W, "eps": cfg.norm_eps, "weight_name": "", "centred": True}, prefix)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m, ff = f"l{i}", layer["mixer"], layer["mlp"]
        parts = {"mixer": _mixer(cfg, layer["type"], m, p + ".mix"), "norm1": norm(p + ".norm1"), "ffn": None, "norm2": None}
        if ff is not None:
            parts["norm2"] = norm(p + ".norm2")
            parts["ffn"] = PartSpec("routed", {
                "hidden_size": W, "experts": ff["experts"], "top": ff["top"], "expert_size": ff["ff"], "activation": "relu2",
                "router": "softmax_groups", "groups": ff["groups"], "keep_groups": ff["keep"], "weight_eps": WEIGHT_SUM_EPS}, p + ".mlp")
        layers.append(LayerSpec("postnorm", parts, cache_of=m.get("kv_from"), params={"alpha": cfg.postln_alpha}))
    spec = ModelSpec(
        hidden_size=W, vocab_size=cfg.vocab, max_position=cfg.max_position,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "weight_name": ""}, "embed"),
        layers=tuple(layers), order=tuple(range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"hidden_size": W, "vocab_size": cfg.vocab, "tied_to": "embed"}, "head"),
        eos_token_id=cfg.eos_token_id,
    )
    spec.validate()
    return spec


register_architecture("Nidorax", NidoraxConfig, build_nidorax_spec)
