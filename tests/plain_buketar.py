"""A plain, slow implementation of the Buketar decoder: whole sequences, no cache, one function
for each mechanism, float64 on the CPU, loops over time where a recurrence says it most plainly.

It shares no code with the package under test: it reads config.json and model.safetensors
itself and states every mechanism from its definition (t: time, h: a sublayer's input).

  norm           n(y) w = y / sqrt(mean(y^2) + eps) * w
  streams        S copies X[0 .. S) of the embedding's output run through the layers; a sublayer reads
                 u = sum_s in[s] X[s], returns y = scale * sublayer(n(u) w) (scale: a value a channel), and then,
                 all from the old streams, X[t] = sum_s mix[s][t] X[s] + out[t] y; the model's last norm reads
                 the sum of the streams
  latent         q = Wq h a head [plain | rotary]; Wdkv h = [c | kr], c normed with a weight; k_a = Wuk_a c,
                 v_a = Wuv_a c; s_ij = (plain parts + turned rotary parts) * scale over j <= i; softmax;
                 the heads times sigmoid(Wg h), an element each; Wo
  rotation       pairs (i, i + r/2) turned by p f_i; with a stretched context the frequencies are blended with
                 f_i / factor and cosine and sine multiplied by 0.1 ln(factor) + 1
  gated linear recurrence   y = gelu(Wy h + b); u = causal filter over time of (Wx h + b), a filter a channel;
                 in equal parts of the channels r = sigmoid(Ra u + b), i = sigmoid(Ri u + b);
                 log a = -8 r softplus(lam); S_t = a S_{t-1} + sqrt(1 - a^2) i u; out = Wo (S y)
  experts        s = sigmoid(Wr h); the ``top`` largest; weights s * scale as they are; an expert:
                 g = min(Wg h, limit), u = clamp(Wu h, -limit, limit), Wd (g sigmoid(1.702 g) (u + 1))
  output         z = head (n(sum of streams) w); cap * tanh(z / cap)
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional, Sequence

import torch

F64 = torch.float64


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    dt = {"F32": torch.float32, "BF16": torch.bfloat16, "F16": torch.float16, "F64": torch.float64,
          "I32": torch.int32, "I64": torch.int64}
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        b, e = info["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[b:e]), dtype=dt[info["dtype"]]).reshape(info["shape"]).clone()
    return out


def load_model_dir(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    w = read_safetensors(os.path.join(model_dir, "model.safetensors"))
    return cfg, {k: v.to(F64) for k, v in w.items()}


# --------------------------------------------------------------------------- small functions
def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# --------------------------------------------------------------------------- rotary positions
def frequencies(rot: dict) -> List[float]:
    """One frequency a pair; ``rot``: base, dims, optionally scaling {factor, original, fast, slow}."""
    n, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return plain

    def pair_with(turns: float) -> float:        # the pair that makes this many turns over the original context
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    first = max(math.floor(pair_with(s["fast"])), 0)
    last = min(math.ceil(pair_with(s["slow"])), n - 1)
    out = []
    for i, f in enumerate(plain):
        slow_share = (i - first) / max(last - first, 0.001)
        slow_share = 0.0 if slow_share < 0 else 1.0 if slow_share > 1 else slow_share
        out.append(slow_share * f / s["factor"] + (1.0 - slow_share) * f)
    return out


def magnitude(rot: dict) -> float:
    s = rot.get("scaling")
    return 0.1 * math.log(s["factor"]) + 1.0 if s else 1.0


def rotate_halves(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, r]: dimension i pairs with i + dims / 2 among the first ``dims``; the rest pass; row t is position t."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    f, mag = frequencies(rot), magnitude(rot)
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(half):
            c, s = mag * math.cos(t * f[i]), mag * math.sin(t * f[i])
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


# --------------------------------------------------------------------------- attention through a latent
def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, dk, rd, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, dk + rd)
    q_plain, q_rot = q[:, :, :dk], rotate_halves(q[:, :, dk:], m.get("rot"))
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :r], w[p + "dkv.norm"], eps)
    k_rot = rotate_halves(down[:, r:].view(T, 1, rd), m.get("rot"))[:, 0]
    k_plain = (c @ w[p + "uk"].T).view(T, H, dk)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    o = torch.zeros((T, H, dv), dtype=F64)
    for a in range(H):
        s = (q_plain[:, a] @ k_plain[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        for i in range(T):
            row = s[i, :i + 1]
            e = torch.exp(row - row.max())
            o[i, a] = (e / e.sum()) @ v[:i + 1, a]
    return (o.reshape(T, H * dv) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# --------------------------------------------------------------------------- gated linear recurrence
def causal_filter(z: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """z [T, C], taps [C, n] (the last column meets the current token), zeros before the start."""
    T, n = z.shape[0], taps.shape[1]
    out = torch.zeros_like(z)
    for t in range(T):
        acc = bias.clone()
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                acc = acc + taps[:, j] * z[src]
        out[t] = acc
    return out


def recurrence_gates(u: torch.Tensor, mats: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """sigmoid of a square matrix a part of the channels: u [T, parts * n], mats [parts, n, n], bias [parts, n]."""
    parts, n, _ = mats.shape
    return torch.cat([sigmoid(u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b]) for b in range(parts)], dim=1)


def gated_recurrence(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    """The states S_1 .. S_T from S_0 = 0."""
    S = torch.zeros(u.shape[1], dtype=F64)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def recurrent_block(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_filter(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = recurrence_gates(u, w[p + "ra"], w[p + "ra.b"])
    i = recurrence_gates(u, w[p + "ri"], w[p + "ri.b"])
    return (gated_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


# --------------------------------------------------------------------------- experts
def clamped_expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def experts_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: dict, forced: Optional[Dict[int, List[int]]] = None) -> torch.Tensor:
    """``forced`` {position: expert ids}: the experts of these tokens are given instead of chosen (their weights are
    still the plain scores): a comparison with a run in fewer bits takes that run's choices where a close call may
    have fallen the other way, so that it measures rounding and not the choice."""
    r = mlp["router"]
    out = torch.zeros_like(h)
    scores = sigmoid(h @ w[p + "router"].T)
    for t in range(h.shape[0]):
        s = scores[t]
        ids = sorted(range(s.shape[0]), key=lambda e: (-s[e].item(), e))[:r["top"]]
        if forced is not None and t in forced:
            ids = list(forced[t])
        for e in ids:
            out[t] += s[e] * r.get("scale", 1.0) * clamped_expert(h[t:t + 1], w, f"{p}e{e}.", mlp["expert"]["limit"])[0]
    return out


# --------------------------------------------------------------------------- streams
def streams_read(X: torch.Tensor, coef: torch.Tensor) -> torch.Tensor:
    """X [S, T, d] -> sum_s coef[s] X[s]."""
    return sum(coef[s] * X[s] for s in range(X.shape[0]))


def streams_join(X: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """mix [from, to]."""
    S = X.shape[0]
    return torch.stack([sum(mix[s, t] * X[s] for s in range(S)) + out[t] * y for t in range(S)])


# --------------------------------------------------------------------------- the model
def running_order(cfg: dict) -> List[int]:
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, k = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * k + list(range(b, n))


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[List[torch.Tensor]] = None,
            forced: Optional[Dict[int, Dict[int, List[int]]]] = None) -> torch.Tensor:
    """Logits [T, V] of one whole sequence; ``layers_out`` collects the sum of the streams after every layer run;
    ``forced`` {layer run: {position: expert ids}}: see ``experts_ff``."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][list(tokens)]
    X = torch.stack([x] * cfg["streams"])
    for run, i in enumerate(running_order(cfg)):
        layer = cfg["layers"][i]
        p = f"l{i}."
        h = rms_norm(streams_read(X, w[p + "hc1.in"]), w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", layer["mixer"], eps)
        elif layer["type"] == "rglru":
            y = recurrent_block(h, w, p + "mix.")
        else:
            raise ValueError(f"layer type {layer['type']!r}")
        X = streams_join(X, y * w[p + "ls1"], w[p + "hc1.mix"], w[p + "hc1.out"])
        if layer.get("mlp") is not None:
            h = rms_norm(streams_read(X, w[p + "hc2.in"]), w[p + "norm2"], eps)
            y = experts_ff(h, w, p + "mlp.", layer["mlp"], None if forced is None else forced.get(run))
            X = streams_join(X, y * w[p + "ls2"], w[p + "hc2.mix"], w[p + "hc2.out"])
        if layers_out is not None:
            layers_out.append(X.sum(dim=0))
    z = rms_norm(X.sum(dim=0), w["final.norm"], eps) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return z if cap is None else cap * torch.tanh(z / cap)
