"""The Tigutar decoder as a ``ModelSpec``: which parts, with which constants and which tensor names.

    x = embed[token]
    a layer:  h = ln(x);  x += residual_mult * (mixer(h) + ff(h))        (ln: layer norm with weight and bias; one for both)
    mixer "attention":  q, k, v without biases; rotary positions on pairs (i, i + dims/2); causal softmax attention whose
              denominator holds a learned term a head; every head times sigmoid(Wg h), one number; Wo.  A layer may read
              another layer's keys and values (``kv_from``) with queries, sink and gate of its own
    mixer "delta":      the gated delta rule (parts/recurrent.py, ``gated_delta_rule``)
    mixer "parallel":   half the sum of two mixers' outputs, each RMS-normed over the width with a weight of its own: windowed
              softmax attention, and gated linear attention (parts/recurrent.py, ``gated_linear_attention``)
    ff "dense":  Wd (silu(Wg h) * (Wu h))
    ff "moe":    sigmoid scores, the ``top`` largest, an expert reads its score times h; clamped gates
    logits = head ln(x)

Tensor names: "embed", "l<i>.norm1" (+ ".b"), "l<i>.mix.{q,k,v,o,g,sink}", "l<i>.mix.{q,k,v}" (+ ".conv"),
"l<i>.mix.{a,b,A_log,dt_bias,g,norm,o}", "l<i>.mix.left.{q,k,v,o,out}", "l<i>.mix.right.{q,k,v,g,o,norm,a1,a2,out}" (a2
+ ".b"), "l<i>.mlp.{gate,up,down}" or "l<i>.mlp.{router,e<j>.{gate,up,down}}", "final.norm" (+ ".b"), "head"; matrices
[out, in].
"""
from __future__ import annotations

from ..config.files import ConfigError
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec
from ..config.tigutar import TigutarConfig

_GATE_ALPHA = 1.702          # an expert's gate is g sigmoid(1.702 g)
_UNIT_EPS = 1e-6             # under the square root of the delta rule's unit vectors


def _attention_spec(d: int, a, p: str, sink_and_gate: bool) -> PartSpec:
    if a.rot is not None:
        position = PartSpec("rope", {"head_dim": a.dim, "rotary_dim": a.rot.dims, "theta": a.rot.base, "pairing": "half"})
    else:
        position = PartSpec("none", {"head_dim": a.dim})
    names = {"q": p + "q", "k": p + "k", "v": p + "v", "o": p + "o", "suffix": ""}
    if sink_and_gate:
        names.update(sink=p + "sink", g=p + "g")
    return PartSpec("gqa_attention", {"hidden_size": d, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim,
                                      "value_dim": a.vdim, "scale": a.scale, "window": a.window, "position": position,
                                      "gate_per_head": sink_and_gate, "shared_keys": a.kv_from is not None, "names": names})


def _delta_spec(d: int, m, p: str, eps: float) -> PartSpec:
    names = {k: p + k for k in ("q", "k", "v", "g", "a", "b", "o", "A_log", "dt_bias", "norm")}
    return PartSpec("gated_delta_rule", {
        "hidden_size": d, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "conv_taps": m.conv,
        "norm_eps": eps, "unit_eps": _UNIT_EPS, "names": dict(names, suffix="", conv_suffix=".conv")})


def _linear_spec(d: int, r, p: str, eps: float, where: str) -> PartSpec:
    if r.decay_rank is None:
        raise ConfigError(f"{where}: the inner width of the decay projection is in no key of config.json; the checkpoint's "
                          "tensor shapes give it, or 'decay_rank' names it")
    names = {k: p + k for k in ("q", "k", "v", "g", "o", "a1", "a2", "norm")}
    return PartSpec("gated_linear_attention", {
        "hidden_size": d, "num_heads": r.heads, "head_dim": r.dim, "value_dim": r.vdim, "decay_rank": r.decay_rank, "tau": r.tau,
        "norm_eps": eps, "names": dict(names, suffix="", bias_suffix=".b")})


def _feed_forward_spec(d: int, f, p: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("gated_mlp", {"hidden_size": d, "intermediate_size": f.ff, "activation": "silu",
                                      "names": {"gate": p + "gate", "up": p + "up", "down": p + "down", "suffix": ""}})
    return PartSpec("moe_mlp", {"hidden_size": d, "expert_size": f.ff, "num_experts": f.experts, "top": f.top, "router_bias": False,
                                "scoring": "sigmoid", "weigh": "input", "activation": "clamped_sigmoid", "limit": f.limit,
                                "alpha": _GATE_ALPHA, "names": {"router": p + "router", "expert": p + "e{e}", "suffix": ""}})


def tigutar_spec(cfg: TigutarConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("layer_norm", {"size": d, "eps": eps, "name": name, "bias_name": name + ".b"})
    layers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        m = l.mixer
        cache_from = None
        if l.type == "attention":
            mixer = _attention_spec(d, m, p + "mix.", sink_and_gate=True)
            cache_from = m.kv_from
        elif l.type == "delta":
            mixer = _delta_spec(d, m, p + "mix.", eps)
        else:
            mixer = PartSpec("parallel_mixers", {
                "left": _attention_spec(d, m.left, p + "mix.left.", sink_and_gate=False),
                "right": _linear_spec(d, m.right, p + "mix.right.", eps, f"layers[{i}].mixer.right"),
                "left_scale": 0.5, "right_scale": 0.5,
                "out_norms": {"left": p + "mix.left.out", "right": p + "mix.right.out", "size": d, "eps": eps}})
        layers.append(LayerSpec(block=PartSpec("parallel_shared_norm", {"residual_scale": cfg.residual_mult}), mixer=mixer,
                                mixer_norm=norm(p + "norm1"), feed_forward_norm=PartSpec("none"),
                                feed_forward=PartSpec("none") if l.mlp is None else _feed_forward_spec(d, l.mlp, p + "mlp."),
                                cache_from=cache_from))
    spec = ModelSpec(
        architecture="Tigutar", vocab_size=cfg.vocab, hidden_size=d, max_position_embeddings=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": d, "name": "embed"}),
        layers=tuple(layers), schedule=tuple(range(len(layers))), final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": d, "name": "head"}))
    spec.validate()
    return spec


TIGUTAR = register_architecture(("Tigutar", "tigutar"), TigutarConfig.from_dict, tigutar_spec,
                                sizes_from_checkpoint=TigutarConfig.with_checkpoint_sizes)
