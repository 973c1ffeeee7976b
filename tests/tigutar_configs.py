"""Small Tigutar configurations for tests, and a writer of random weights for them.

The configurations differ from one another in every size and option: every kind of mixer first, last and in the middle;
attention heads over one, some and as many key/value heads; key heads narrower than, wider than and equal to value heads,
among them the widths that the tensor-core kernels take in every combination; rotation of a part of a head, of all of it
and none; windows shorter and longer than a page; layers that read another layer's keys, one of them directly behind and
one with other layers between; delta layers with fewer query/key heads than heads and as many, 1 to 5 taps; decay
projections 3 to 16 wide; experts with top = 1, some and all; layers without a feed-forward; widths that are and are not
multiples of 8.

Weights are drawn so that faults show: queries and keys large enough that attention is far from uniform, sinks of both
signs up to the largest scores, router logits of standard deviation 1.5, decays from a memory of hundreds of tokens to a
few, step sizes over the whole of (0, 1).  They are stored in bfloat16, so a 32-bit run and a bfloat16 run compute on the
same numbers.

``router_std``: the standard deviation of the router's logits (see ``besuzen_configs``: the bfloat16 runs of subprocesses
draw decisive routers).
"""
import json
import math
import os

import torch

from rustyllm_b200.weights.safetensors_io import write_safetensors


def att(heads, kv_heads, dim, vdim, scale, rot=None, window=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def attention(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def parallel(left, heads, dim, vdim, tau, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def model(vocab, width, eps, mult, layers):
    return {"architecture": "Tigutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


# the inner width of the decay projections is in no key of config.json (the tensors' shapes give it): per configuration
DECAY_RANK = {"A": 5, "B": 3, "C": 16, "D": 8}

CONFIGS = {
    # narrow heads (the any-shape attention kernel): a delta layer first, attention whose values are narrower than its keys and
    # half of whose head is rotated, a layer on its keys with more heads, a window shorter than a page
    "A": model(97, 72, 1e-5, 0.4, [
        delta(4, 2, 24, 16, 4, moe(6, 2, 16, 1.2)),
        attention(att(4, 2, 16, 8, 0.3, rot=(8, 10000.0)), dense(48)),
        parallel(att(3, 1, 12, 20, 0.35, rot=(12, 500.0), window=19), 3, 16, 12, 8.0, None),
        attention(att(6, 2, 16, 8, 0.35, rot=(8, 10000.0), kv_from=1), moe(5, 1, 24, 0.8))]),
    # a width that is no multiple of 8 (no tensor-core product takes it); one tap (nothing is kept), a layer on the keys of the
    # one directly in front, no rotation, all experts chosen, a window of one page exactly, state rows that are no multiple of 4
    "B": model(53, 44, 1e-6, 1.0, [
        attention(att(2, 2, 12, 12, 0.4), moe(3, 3, 12, 2.0)),
        attention(att(2, 2, 12, 12, 0.3, kv_from=0), None),
        delta(3, 3, 18, 10, 1, dense(20)),
        parallel(att(2, 2, 8, 24, 0.4, rot=(4, 100.0), window=64), 1, 22, 14, 3.0, moe(4, 2, 8, 1.0))]),
    # the widths that the tensor-core attention kernels take: keys of 64 with values of 128 under a window across pages, keys of
    # 128 with values of 64, both equal; a layer on others' keys with other layers between, a delta layer with heads of 64
    "C": model(211, 128, 1e-5, 0.55, [
        parallel(att(4, 2, 64, 128, 0.125, rot=(64, 300000.0), window=100), 4, 32, 24, 16.0, moe(8, 3, 32, 1.5)),
        attention(att(4, 1, 128, 64, 0.09, rot=(64, 10000.0)), dense(96)),
        delta(4, 1, 64, 32, 3, dense(64)),
        attention(att(2, 2, 64, 64, 0.125, rot=(32, 20000.0)), moe(8, 1, 40, 1.0)),
        attention(att(8, 1, 128, 64, 0.09, rot=(64, 10000.0), kv_from=1), moe(4, 2, 24, 0.7))]),
    # wide heads of the recurrences (more than 128 rows), keys and values of 128 with a window longer than two pages
    "D": model(150, 80, 1e-5, 0.25, [
        delta(2, 1, 136, 40, 5, None),
        parallel(att(2, 1, 128, 128, 0.08, rot=(128, 50000.0), window=150), 2, 160, 20, 20.0, dense(40)),
        parallel(att(2, 2, 64, 64, 0.12, rot=(48, 1000.0), window=33), 2, 72, 36, 5.0, moe(5, 5, 16, 3.0))]),
}


def tensor_shapes(cfg: dict, rank: int) -> dict:
    d, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, d), "final.norm": (d,), "final.norm.b": (d,), "head": (V, d)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"] = out[p + "norm1.b"] = (d,)

        def att_shapes(q, m):
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out[q + "q"] = (H * dk, d)
            if m.get("kv_from") is None:
                out.update({q + "k": (G * dk, d), q + "v": (G * dv, d)})
            out[q + "o"] = (d, H * dv)
        q = p + "mix."
        if l["type"] == "attention":
            att_shapes(q, m)
            out.update({q + "sink": (m["heads"],), q + "g": (m["heads"], d)})
        elif l["type"] == "delta":
            H, G, dk, dv, t = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            out.update({q + "q": (G * dk, d), q + "q.conv": (G * dk, t), q + "k": (G * dk, d), q + "k.conv": (G * dk, t),
                        q + "v": (H * dv, d), q + "v.conv": (H * dv, t), q + "b": (H, d), q + "a": (H, d), q + "A_log": (H,),
                        q + "dt_bias": (H,), q + "norm": (dv,), q + "g": (H * dv, d), q + "o": (d, H * dv)})
        else:
            att_shapes(q + "left.", m["left"])
            r = m["right"]
            H, dk, dv = r["heads"], r["dim"], r["vdim"]
            q += "right."
            out.update({q + "q": (H * dk, d), q + "k": (H * dk, d), q + "v": (H * dv, d), q + "g": (H * dv, d), q + "o": (d, H * dv),
                        q + "norm": (dv,), q + "a1": (rank, d), q + "a2": (H * dk, rank), q + "a2.b": (H * dk,), q + "out": (d,),
                        p + "mix.left.out": (d,)})
        mlp, q = l["mlp"], p + "mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            out.update({q + "gate": (mlp["ff"], d), q + "up": (mlp["ff"], d), q + "down": (d, mlp["ff"])})
        else:
            F = mlp["expert"]["ff"]
            out[q + "router"] = (mlp["router"]["experts"], d)
            for e in range(mlp["router"]["experts"]):
                out.update({f"{q}e{e}.gate": (F, d), f"{q}e{e}.up": (F, d), f"{q}e{e}.down": (d, F)})
    return out


def draw_weights(cfg: dict, rank: int, seed: int, router_std: float = 1.5) -> dict:
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        last = name.rsplit(".", 1)[-1]

        def normal(std):
            return torch.randn(shape, generator=g, dtype=torch.float64) * std

        def uniform(lo, hi):
            return lo + (hi - lo) * torch.rand(shape, generator=g, dtype=torch.float64)
        kind = cfg["layers"][int(name[1:name.index(".")])]["type"] if name[0] == "l" else None
        if last in ("norm1", "norm", "out"):
            t = 1.0 + normal(0.15)
        elif name.endswith("a2.b"):
            t = uniform(-3.0, 6.0)                   # decays from a few tokens to a few thousand
        elif last == "b" and len(shape) == 1:        # the biases of the layer norms
            t = normal(0.3)
        elif last == "b":
            t = normal(2.0 / math.sqrt(shape[1]))
        elif last == "sink":
            t = uniform(-2.0, 4.0)
        elif last == "A_log":
            t = uniform(-4.0, 1.0)
        elif last == "dt_bias":
            t = uniform(-2.0, 1.0)
        elif last == "conv":
            t = normal(0.6)
        elif last == "router":
            t = normal(router_std / math.sqrt(shape[1]))
        elif name == "embed":
            t = normal(1.0)
        elif last in ("q", "k") and ".right." not in name and kind != "delta":
            t = normal(2.0 / math.sqrt(shape[1]))        # sharp attention
        elif last in ("gate", "up") and ".e" in name:
            t = normal(2.0 / math.sqrt(shape[1]))        # clamps that act
        else:
            t = normal(1.0 / math.sqrt(shape[-1]))
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(name: str, model_dir: str, seed: int = 0, cfg: dict = None, rank: int = None, router_std: float = 1.5) -> str:
    cfg = CONFIGS[name] if cfg is None else cfg
    rank = DECAY_RANK[name] if rank is None else rank
    os.makedirs(model_dir, exist_ok=True)
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(model_dir, "model.safetensors"), draw_weights(cfg, rank, seed, router_std))
    return model_dir


def random_config(seed: int):
    """A configuration with every size drawn: (config, decay rank)."""
    r = torch.Generator().manual_seed(2000 + seed)

    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=r))]
    d = pick(24, 36, 40, 50, 64, 72)

    def rand_att(window_ok):
        G = pick(1, 2, 3)
        dk, dv = pick(8, 12, 16, 32, 64), pick(8, 16, 24, 64, 128)
        rot = (pick(4, 8, dk), pick(100.0, 10000.0, 300000.0)) if pick(0, 1, 1) else None
        return att(G * pick(1, 2, 3), G, dk, dv, 1.0 / math.sqrt(dk), rot=rot, window=pick(5, 16, 63, 65, 128) if window_ok else None)

    def rand_mlp():
        kind = pick("dense", "moe", "moe", None)
        if kind is None:
            return None
        if kind == "dense":
            return dense(pick(16, 40, 56))
        E = pick(1, 2, 3, 5, 9)
        return moe(E, pick(*range(1, E + 1)), pick(8, 16, 24), pick(0.6, 1.5, 4.0))
    layers, owners = [], []
    for i in range(pick(3, 4, 5)):
        kind = pick("attention", "attention", "delta", "parallel")
        if kind == "attention":
            if owners and pick(0, 1):
                j = pick(*owners)
                m = dict(layers[j]["mixer"], kv_from=j, scale=pick(0.2, 0.35))
                m["heads"] = m["kv_heads"] * pick(1, 2, 4)
                layers.append(attention(m, rand_mlp()))
            else:
                owners.append(i)
                layers.append(attention(rand_att(False), rand_mlp()))
        elif kind == "delta":
            G = pick(1, 2, 3)
            layers.append(delta(G * pick(1, 2), G, pick(6, 8, 16, 33, 64), pick(8, 10, 24, 40), pick(1, 2, 3, 4, 6), rand_mlp()))
        else:
            layers.append(parallel(rand_att(True), pick(1, 2, 3), pick(6, 8, 16, 40), pick(8, 12, 24), pick(1.0, 4.0, 16.0), rand_mlp()))
    return model(pick(31, 64, 150), d, pick(1e-5, 1e-6), pick(0.2, 0.35, 0.5), layers), pick(2, 4, 8)
