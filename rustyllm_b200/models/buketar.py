"""The Buketar decoder as a ``ModelSpec``: which parts, with which constants and which tensor names.

    X = ``streams`` copies of embed[token]
    a sublayer:  u = sum_s in[s] X[s];  y = ls * sublayer(rms_norm(u) * norm);  X[t] = sum_s mix[s, t] X[s] + out[t] y
              (a layer: the mixer, then the feed-forward where it has one; parts/streams.py)
    mixer "rglru":             a gelu branch times a gated linear recurrence of one state a channel behind a short causal
                               filter (parts/recurrent.py, ``gated_linear_recurrence``)
    mixer "latent_attention":  keys and values from one normed latent a token plus one rotary key part for all heads;
                               queries straight from the input; half-split rotary pairs, stretched frequencies where
                               the file says so; an output gate an element (parts/latent.py)
    ff "moe": sigmoid scores, the largest chosen, their scores times a constant as weights (not renormalised); experts
              Wd (g sigmoid(1.702 g) (u + 1)) with g = min(Wg h, limit), u = clamp(Wu h, -limit, limit)
    the layers of the loop run several times in a row, every pass with a cache or state of its own
    logits = cap * tanh(head (rms_norm(sum_s X[s]) * final.norm) / cap)

Tensor names: "embed", "l<i>.norm1", "l<i>.norm2", "l<i>.ls1", "l<i>.ls2", "l<i>.hc1.{in,out,mix}", "l<i>.hc2.{in,out,mix}",
"l<i>.mix.{y,x,conv,ra,ri}" (+ ".b"), "l<i>.mix.{lam,o}" or "l<i>.mix.{q,dkv,dkv.norm,uk,uv,g,o}",
"l<i>.mlp.{router,e<j>.{gate,up,down}}", "final.norm", "head"; matrices [out, in].
"""
from __future__ import annotations

from ..config.buketar import BuketarConfig
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec

DECAY_RATE = 8.0         # log a = -8 r softplus(lam)
GATE_ALPHA = 1.702       # the experts' gate: g sigmoid(1.702 g)


def _position(head_dim: int, rot) -> PartSpec:
    if rot is None:
        return PartSpec("none", {"head_dim": head_dim})
    params = {"head_dim": head_dim, "rotary_dim": rot.dims, "base": rot.base}
    if rot.scaling is not None:
        params.update(rot.scaling.to_dict())
    return PartSpec("rope_yarn", params)


def buketar_spec(cfg: BuketarConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    layers, ignored = [], []
    for i, l in enumerate(cfg.layers):
        p, q = f"l{i}.", f"l{i}.mix."
        m = l.mixer
        if l.type == "rglru":
            mixer = PartSpec("gated_linear_recurrence", {
                "hidden_size": d, "width": m.width, "blocks": m.blocks, "conv_taps": m.conv, "decay_rate": DECAY_RATE,
                "names": {"y": q + "y", "x": q + "x", "conv": q + "conv", "ra": q + "ra", "ri": q + "ri", "lam": q + "lam", "o": q + "o",
                          "suffix": "", "bias_suffix": ".b"}})
        else:
            mixer = PartSpec("latent_attention", {
                "hidden_size": d, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim,
                "q_rank": None, "kv_rank": m.kv_rank, "scale": m.scale, "norm_eps": eps, "head_gate": False, "element_gate": True,
                "position": _position(m.rot_dim or 2, m.rot),
                "names": {"q": q + "q", "dkv": q + "dkv", "dkv_norm": q + "dkv.norm", "uk": q + "uk", "uv": q + "uv", "g": q + "g",
                          "o": q + "o", "suffix": ""}})
        names = {"mixer": p + "hc1.", "mixer_scale": p + "ls1", "feed_forward": p + "hc2.", "feed_forward_scale": p + "ls2"}
        if l.mlp is None:
            ff, ff_norm = PartSpec("none"), PartSpec("none")
            ignored += [p + "norm2", p + "ls2", p + "hc2.in", p + "hc2.out", p + "hc2.mix"]
        else:
            f = l.mlp
            ff = PartSpec("moe_mlp", {
                "hidden_size": d, "expert_size": f.ff, "num_experts": f.experts, "top": f.top, "router_bias": False,
                "scoring": "sigmoid", "weight_scale": f.scale, "activation": "clamped_sigmoid", "limit": f.limit, "alpha": GATE_ALPHA,
                "names": {"router": p + "mlp.router", "expert": p + "mlp.e{e}", "suffix": ""}})
            ff_norm = PartSpec("rms_norm", {"size": d, "eps": eps, "name": p + "norm2"})
        layers.append(LayerSpec(block=PartSpec("hyper_connected", {"hidden_size": d, "streams": cfg.streams, "names": names}),
                                mixer=mixer, mixer_norm=PartSpec("rms_norm", {"size": d, "eps": eps, "name": p + "norm1"}),
                                feed_forward=ff, feed_forward_norm=ff_norm))
    spec = ModelSpec(
        architecture="Buketar", vocab_size=cfg.vocab, hidden_size=d, max_position_embeddings=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": d, "name": "embed"}),
        layers=tuple(layers), schedule=cfg.schedule(),
        final_norm=PartSpec("rms_norm", {"size": d, "eps": eps, "name": "final.norm"}),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": d, "name": "head", "softcap": cfg.logit_softcap}),
        ignored_tensors=tuple(ignored), streams=cfg.streams)
    spec.validate()
    return spec


BUKETAR = register_architecture(("Buketar", "buketar"), BuketarConfig.from_dict, buketar_spec)
