"""Kepevik laid out as a ModelSpec: a decoder whose config lists its layers one by one.

The embedding is scaled by a constant.  Every sublayer has an RMS norm before it and one on its output, both with weights stored
around zero, and a learned vector on the normed output: x <- x + scale * norm_b(sublayer(norm(x))).  The mixer is
  mlstm     a matrix memory per head with exponential input gates and sigmoid forget gates under a running maximum, the read-out
            divided by a normaliser; an RMS norm per head and a sigmoid gate;
  parallel  a causal attention whose values are its keys before rotation, beside a delta rule with a decay per key channel
            through a low rank and a sigmoid gate through another; the two summed with two constants.
The feed-forward is a dense one with biases (gelu), or a mixture of gated experts: softmax scores over all experts, a correction
that enters the choice only, the scores themselves as weights, experts that pass the input through, and a shared expert behind a
gate of one number per token; or absent.  The logits are the normed stream times the embedding table.  Tensors: `embed`,
`l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`.
"""
from __future__ import annotations

from ..config.model_config import KepevikConfig, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec

UNIT_EPS = 1e-6             # added to the sums of squares under the delta rule's unit norms


def _mixer(cfg: KepevikConfig, kind: str, m: dict, prefix: str) -> PartSpec:
    W, eps = cfg.width, cfg.norm_eps
    if kind == "mlstm":
        return PartSpec("mlstm", {"hidden_size": W, "num_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
                                  "gate_cap": m["gate_cap"], "eps": eps}, prefix)
    a, b = m["left"], m["right"]
    left = PartSpec("attention", {
        "hidden_size": W, "num_heads": a["heads"], "num_kv_heads": a["kv_heads"], "head_dim": a["dim"], "scale": a["scale"],
        "position": PartSpec("rope_pairs", {"dims": a["rot_dims"], "base": a["rot_base"], "layout": "halves"}),
        "keys_as_values": True, "names": {"q": "q", "k": "k", "o": "o"}}, prefix + ".left")
    right = PartSpec("gated_delta", {"hidden_size": W, "num_heads": b["heads"], "num_qk_heads": b["kv_heads"], "head_dim": b["dim"],
                                     "value_dim": b["vdim"], "taps": b["conv"], "eps": eps, "unit_eps": UNIT_EPS,
                                     "channel_decay": True, "low_rank_gate": True, "rank": b["dim"]}, prefix + ".right")
    return PartSpec("parallel", {"hidden_size": W, "left": left, "right": right, "combine": "scaled_sum",
                                 "left_scale": m["left_scale"], "right_scale": m["right_scale"]}, prefix)


def _ffn(cfg: KepevikConfig, ff: dict, prefix: str) -> PartSpec:
    W = cfg.width
    if ff["kind"] == "dense":
        return PartSpec("mlp", {"hidden_size": W, "intermediate_size": ff["ff"], "activation": "gelu", "bias": True}, prefix)
    return PartSpec("routed", {"hidden_size": W, "experts": ff["experts"], "identity": ff["identity"], "top": ff["top"],
                               "expert_size": ff["ff"], "activation": "silu", "gated": True, "router": "softmax_corrected",
                               "shared_size": ff["shared"], "shared_gated": True, "shared_gate": True}, prefix)


def build_kepevik_spec(cfg: KepevikConfig) -> ModelSpec:
    W = cfg.width

    def norm(prefix, weight_name="", scale_name=None):
        return PartSpec("rmsnorm", {"size": W, "eps": cfg.norm_eps, "weight_name": weight_name, "centred": True,
                                    "scale_name": scale_name}, prefix)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, ff = f"l{i}", layer["mlp"]
        parts = {"norm1": norm(p, "norm1"), "mixer": _mixer(cfg, layer["type"], layer["mixer"], p + ".mix"),
                 "post1": norm(p, "norm1b", "ls1"), "norm2": None, "ffn": None, "post2": None}
        if ff is not None:
            parts.update({"norm2": norm(p, "norm2"), "ffn": _ffn(cfg, ff, p + ".mlp"), "post2": norm(p, "norm2b", "ls2")})
        layers.append(LayerSpec("sandwich", parts))
    spec = ModelSpec(
        hidden_size=W, vocab_size=cfg.vocab, max_position=cfg.max_position,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "weight_name": "",
                                               "scale": cfg.embedding_scale}, "embed"),
        layers=tuple(layers), order=tuple(range(len(layers))), final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"hidden_size": W, "vocab_size": cfg.vocab, "tied_to": "embed"}, "head"),
        eos_token_id=cfg.eos_token_id,
    )
    spec.validate()
    return spec


register_architecture("Kepevik", KepevikConfig, build_kepevik_spec)
