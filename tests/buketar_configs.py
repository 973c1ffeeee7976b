"""Small Buketar configurations for tests, and a writer of random weights for them.

The configurations differ from one another in every size and option: one stream, some and more than eight; a loop over
several layers, over the first one alone, and none; recurrent layers first and last, latent layers first and last;
recurrences whose parts are one block, several, of even and of odd width (and of widths the tensor-core products cannot
address); filters of one tap to five; latents narrower than the heads together and wider, key rows that are and are not
multiples of 16, rotary parts of 6 to 32 dimensions with plain and with stretched frequencies, more than 16 heads, value
heads narrower and wider than key heads; one expert a token, some, all; router factors of 1 and others; layers without a
feed-forward; widths that are and are not multiples of 8 and of 4; logits with and without a soft cap.

Weights are drawn so that faults show: queries and keys large enough that attention is far from uniform, decays that
reach from a memory of thousands of tokens to a few, gates' sums of standard deviation 1, experts' gate and up values
that meet the limit on either side, mixing matrices near the identity with noise on every element (so that [from, to]
and [to, from] differ), factors a channel and a stream that are all different.  They are stored in bfloat16, so a 32-bit
run and a bfloat16 run compute on the same numbers.

``router_std``: the standard deviation of the router's logits, 1.5: lively routers whose scores often lie close
together.  The bfloat16 engine tests hand the run's own choices to the plain implementation (a close call that falls
the other way once the router's input is rounded is no fault of a kernel); the 32-bit runs are compared as they are.
"""
import json
import math
import os

import torch

from rustyllm_b200.weights.safetensors_io import write_safetensors


def rglru(width, blocks, conv, mlp):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, mlp, base=10000.0, scaling=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": rot}}


def moe(experts, top, ff, limit, scale=None):
    r = {"experts": experts, "top": top}
    if scale is not None:
        r["scale"] = scale
    return {"kind": "moe", "router": r, "expert": {"ff": ff, "limit": limit}}


CONFIGS = {
    # three streams; the loop runs a recurrent and a latent layer three times; stretched frequencies
    "A": {"architecture": "Buketar", "vocab": 101, "width": 64, "norm": {"eps": 1e-5}, "streams": 3, "logit_softcap": 12.0,
          "loop": {"start": 1, "stop": 3, "times": 3},
          "layers": [rglru(48, 3, 4, moe(6, 2, 24, 0.9, 1.2)),
                     latent(4, 16, 8, 24, 40, 0.11, moe(5, 1, 16, 1.3, 1.5), base=500.0, scaling=(8.0, 64, 8.0, 1.0)),
                     rglru(32, 1, 3, moe(4, 2, 16, 0.6)),
                     rglru(64, 2, 2, None)]},
    # a width that is no multiple of 8 and odd parts: no tensor-core product takes them; one stream, no loop, no soft cap,
    # plain frequencies, all experts chosen, filters of one tap and five
    "B": {"architecture": "Buketar", "vocab": 53, "width": 44, "norm": {"eps": 1e-6}, "streams": 1,
          "layers": [latent(3, 10, 6, 12, 20, 0.4, moe(3, 3, 12, 2.0)),
                     rglru(21, 3, 5, None),
                     rglru(44, 4, 1, moe(7, 2, 20, 0.5, 0.6)),
                     latent(1, 12, 2, 8, 12, 0.5, None, base=100.0)]},
    # the tensor-core kernels throughout: key rows of 96 and 144, more than 16 heads, two streams, the first layer alone
    # twice, one expert a token
    "C": {"architecture": "Buketar", "vocab": 211, "width": 128, "norm": {"eps": 1e-5}, "streams": 2, "logit_softcap": 30.0,
          "loop": {"start": 0, "stop": 1, "times": 2},
          "layers": [rglru(192, 2, 4, moe(8, 1, 32, 1.0, 2.0)),
                     latent(20, 16, 32, 16, 64, 0.2, moe(6, 4, 24, 0.8, 1.5), base=1.0e5, scaling=(16.0, 128, 16.0, 2.0)),
                     rglru(128, 8, 4, moe(16, 2, 16, 1.5, 1.2)),
                     latent(5, 64, 16, 32, 128, 0.125, moe(4, 2, 40, 1.0), base=1.0e6, scaling=(2.0, 100, 4.0, 1.0))]},
    # a width that is no multiple of 4, nine streams (more than the fixed forms have), the whole model twice
    "D": {"architecture": "Buketar", "vocab": 64, "width": 50, "norm": {"eps": 1e-4}, "streams": 9, "logit_softcap": 8.0,
          "loop": {"start": 0, "stop": 2, "times": 2},
          "layers": [latent(2, 24, 16, 16, 48, 0.25, moe(9, 3, 8, 0.7, 3.0), scaling=(4.0, 32, 32.0, 1.0)),
                     rglru(40, 1, 4, moe(2, 1, 18, 1.1))]},
}


def running_layers(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def tensor_shapes(cfg: dict) -> dict:
    d, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    out = {"embed": (V, d), "final.norm": (d,), "head": (V, d)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q = p + "mix."
        for k in ((1, 2) if l["mlp"] is not None else (1,)):
            out.update({f"{p}norm{k}": (d,), f"{p}ls{k}": (d,), f"{p}hc{k}.in": (S,), f"{p}hc{k}.out": (S,), f"{p}hc{k}.mix": (S, S)})
        if l["type"] == "rglru":
            W, b = m["width"], m["blocks"]
            n = W // b
            out.update({q + "y": (W, d), q + "y.b": (W,), q + "x": (W, d), q + "x.b": (W,), q + "conv": (W, m["conv"]), q + "conv.b": (W,),
                        q + "ra": (b, n, n), q + "ra.b": (b, n), q + "ri": (b, n, n), q + "ri.b": (b, n), q + "lam": (W,), q + "o": (d, W)})
        else:
            H, r = m["heads"], m["kv_rank"]
            out.update({q + "q": (H * (m["dim"] + m["rot_dim"]), d), q + "dkv": (r + m["rot_dim"], d), q + "dkv.norm": (r,),
                        q + "uk": (H * m["dim"], r), q + "uv": (H * m["vdim"], r), q + "g": (H * m["vdim"], d), q + "o": (d, H * m["vdim"])})
        if l["mlp"] is not None:
            F = l["mlp"]["expert"]["ff"]
            out[p + "mlp.router"] = (l["mlp"]["router"]["experts"], d)
            for e in range(l["mlp"]["router"]["experts"]):
                x = f"{p}mlp.e{e}."
                out.update({x + "gate": (F, d), x + "up": (F, d), x + "down": (d, F)})
    return out


def draw_weights(cfg: dict, seed: int, router_std: float = 1.5) -> dict:
    g = torch.Generator().manual_seed(seed)
    out = {}
    S = cfg["streams"]
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]

        def normal(std):
            return torch.randn(shape, generator=g, dtype=torch.float64) * std

        def uniform(lo, hi):
            return lo + (hi - lo) * torch.rand(shape, generator=g, dtype=torch.float64)
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + normal(0.15)
        elif last in ("ls1", "ls2"):
            t = uniform(0.4, 1.0)
        elif last == "in":
            t = uniform(0.5, 1.5) / S
        elif last == "out":
            t = uniform(0.4, 1.2)
        elif last == "mix":
            t = torch.eye(S, dtype=torch.float64) * 0.9 + normal(0.15 / math.sqrt(S))
        elif last == "b":
            t = normal(0.3)
        elif last == "lam":
            t = uniform(-9.0, 1.0)
        elif last in ("ra", "ri"):
            t = normal(1.0 / math.sqrt(shape[2]))
        elif last == "conv":
            t = normal(1.0 / math.sqrt(shape[1]))
        elif last == "router":
            t = normal(router_std / math.sqrt(shape[1]))
        elif name == "embed":
            t = normal(1.0)
        elif last == "q":
            t = normal(2.5 / math.sqrt(shape[1]))        # sharp attention
        else:
            t = normal(1.0 / math.sqrt(shape[-1]))
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(model_dir: str, cfg: dict, seed: int = 0, weights: dict = None) -> str:
    os.makedirs(model_dir, exist_ok=True)
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(model_dir, "model.safetensors"), draw_weights(cfg, seed) if weights is None else weights)
    return model_dir


def random_config(seed: int) -> dict:
    """A configuration with every size drawn."""
    r = torch.Generator().manual_seed(4000 + seed)

    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=r))]

    def rand_mlp():
        if pick(0, 1, 1, 1) == 0:
            return None
        E = pick(1, 2, 3, 5, 8)
        return moe(E, pick(*range(1, E + 1)), pick(8, 10, 16, 24), pick(0.5, 1.0, 3.0), pick(None, 1.0, 1.6, 2.5))

    def rand_layer():
        if pick(0, 1):
            b = pick(1, 2, 3, 5)
            return rglru(b * pick(5, 8, 12, 16), b, pick(1, 2, 3, 4, 6), rand_mlp())
        dk, rd = pick(6, 8, 16, 24), pick(4, 8, 16)
        scaling = pick(None, (4.0, 48, 16.0, 1.0), (10.0, 200, 32.0, 2.0), (1.5, 20, 2.0, 1.0))
        return latent(pick(1, 2, 3, 7, 16, 18), dk, rd, pick(8, 10, 16, 32), pick(12, 24, 32, 48), 1.0 / math.sqrt(dk + rd), rand_mlp(),
                      base=pick(100.0, 10000.0, 500000.0), scaling=scaling)
    layers = [rand_layer() for _ in range(pick(1, 2, 3, 4))]
    cfg = {"architecture": "Buketar", "vocab": pick(31, 64, 150), "width": pick(24, 36, 40, 50, 64, 72), "norm": {"eps": pick(1e-5, 1e-6)},
           "streams": pick(1, 2, 3, 4, 5), "layers": layers}
    if pick(0, 1):
        a = pick(*range(len(layers)))
        cfg["loop"] = {"start": a, "stop": pick(*range(a + 1, len(layers) + 1)), "times": pick(1, 2, 3)}
    if pick(0, 1):
        cfg["logit_softcap"] = pick(5.0, 20.0, 50.0)
    return cfg
