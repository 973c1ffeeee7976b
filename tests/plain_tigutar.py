"""A plain, slow implementation of the Tigutar decoder: whole sequences, no cache, one function for each mechanism,
float64 on the CPU, loops over time where a recurrence says it most plainly.

It shares no code with the package under test: it reads config.json and model.safetensors itself and states every
mechanism from its definition (t: time, h: a sublayer's input).

  layer norm   ln(y) = (y - mean(y)) / sqrt(mean((y - mean(y))^2) + eps) * w + b
  rms norm     rms(y) = y / sqrt(mean(y^2) + eps) * w
  layer        h = ln(x);  x += m (mixer(h) + ff(h))                       (one norm, read by both)
  attention    q, k, v = W h; rotation of pairs (i, i + dims/2) of the first ``dims`` dimensions of q and k;
               s_ij = (q_i . k_j) scale for visible j; a softmax whose denominator may hold one more term exp(sink_h);
               optionally the head times sigmoid((Wg h)_h); Wo.  A layer may use another layer's rotated keys and
               values with queries of its own
  delta rule   q, k, v = silu(filter(W h)); q, k divided by sqrt(sum of squares + 1e-6), q times dim^-1/2;
               b = sigmoid(Wb h), g = exp(-exp(A) softplus(Wa h + dt_bias)) a head;
               S = g S;  u = b (v - S^T k);  S = S + k u^T;  o = S^T q;  Wo (rms per head(o) * silu(Wg h))
  linear       q = dim^-1/2 Wq h, k, v = W h; a = sigmoid(W2 (W1 h) + c)^(1/tau) a head and key channel;
               S = diag(a) S + k v^T;  o = S^T q;  Wo (rms per head(o) * silu(Wg h))
  side by side (rms_left(attention(h)) + rms_right(linear(h))) / 2          (over the model's width)
  dense ff     Wd (silu(Wg h) * (Wu h))
  experts      s = sigmoid(Wr h); the ``top`` largest; each reads s_e h: g = min(Wg y, L), u = clamp(Wu y, -L, L),
               Wd (g sigmoid(1.702 g) (u + 1)); their plain sum
  output       head (ln(x))
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
def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w + b


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def unit_vector(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def causal_filter(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [T, C], taps [C, n]: y_t = sum_j taps[:, j] u_{t - (n - 1) + j}; zeros before the start."""
    T, C = u.shape
    n = taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


# --------------------------------------------------------------------------- attention
def rotate_halves(x: torch.Tensor, positions: Sequence[int], dims: int, base: float) -> torch.Tensor:
    """x [T, heads, dim]: dimension i pairs with i + dims/2 among the first ``dims``; the rest pass."""
    out = x.clone()
    half = dims // 2
    for t, p in enumerate(positions):
        for i in range(half):
            a = p * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: Optional[int] = None,
                      sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; query head h reads key/value head h // (H / G); position i
    sees j <= i, with a window only i - j < window; ``sink`` [H]: exp(sink_h) more in the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        for i in range(T):
            lo = 0 if window is None else max(0, i - window + 1)
            row = s[i, lo:i + 1]
            top = row.max()
            if sink is not None:
                top = torch.maximum(top, sink[h])
            p = torch.exp(row - top)
            total = p.sum()
            if sink is not None:
                total = total + torch.exp(sink[h] - top)
            out[i, h] = (p / total) @ v[lo:i + 1, g]
    return out


def attention_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, shared=None):
    """The attention of a layer; ``shared``: the (rotated keys, values) of the layer it reads.  Sink and gate where the
    layer has their tensors.  Returns (output [T, d], (keys, values))."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot")

    def turn(x):
        return rotate_halves(x, range(T), rot["dims"], rot["base"]) if rot and rot.get("dims") else x
    q = turn((h @ w[p + "q"].T).view(T, H, dk))
    if shared is None:
        shared = (turn((h @ w[p + "k"].T).view(T, G, dk)), (h @ w[p + "v"].T).view(T, G, dv))
    k, v = shared
    mask = m.get("mask")
    o = softmax_attention(q, k, v, m["scale"], mask["size"] if mask else None, w.get(p + "sink"))
    if p + "g" in w:
        o = o * sigmoid(h @ w[p + "g"].T).view(T, H, 1)
    return o.reshape(T, H * dv) @ w[p + "o"].T, shared


# --------------------------------------------------------------------------- recurrences with a matrix state a head
def delta_scan(q, k, v, g, beta, state=None):
    """One head: q, k [T, dk], v [T, dv], g, beta [T] -> (o [T, dv], last state [dk, dv])."""
    T, dk = q.shape
    S = torch.zeros((dk, v.shape[1]), dtype=F64) if state is None else state.clone()
    o = torch.zeros((T, v.shape[1]), dtype=F64)
    for t in range(T):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o, S


def delta_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def projected(name):
        return silu(causal_filter(h @ w[p + name].T, w[p + name + ".conv"]))
    q = unit_vector(projected("q").view(T, G, dk)) * dk ** -0.5
    k = unit_vector(projected("k").view(T, G, dk))
    v = projected("v").view(T, H, dv)
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = torch.zeros((T, H, dv), dtype=F64)
    for hd in range(H):
        gq = hd // (H // G)
        o[:, hd], _ = delta_scan(q[:, gq], k[:, gq], v[:, hd], g[:, hd], beta[:, hd])
    o = rms_norm(o, w[p + "norm"], eps) * silu(h @ w[p + "g"].T).view(T, H, dv)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def linear_scan(q, k, v, a, state=None):
    """One head: q, k, a [T, dk], v [T, dv] -> (o [T, dv], last state [dk, dv])."""
    T, dk = q.shape
    S = torch.zeros((dk, v.shape[1]), dtype=F64) if state is None else state.clone()
    o = torch.zeros((T, v.shape[1]), dtype=F64)
    for t in range(T):
        S = a[t].unsqueeze(1) * S + torch.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o, S


def linear_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, dk) * dk ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, dk)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    a = (sigmoid(z) ** (1.0 / m["tau"])).view(T, H, dk)
    o = torch.zeros((T, H, dv), dtype=F64)
    for hd in range(H):
        o[:, hd], _ = linear_scan(q[:, hd], k[:, hd], v[:, hd], a[:, hd])
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * dv) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# --------------------------------------------------------------------------- feed-forwards
def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(scores: torch.Tensor, top: int) -> List[int]:
    return sorted(range(scores.shape[0]), key=lambda e: (-scores[e].item(), e))[:top]


def experts_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: dict, forced: Optional[Dict[int, List[int]]] = None) -> torch.Tensor:
    """``forced`` {position: expert ids}: the experts of these tokens are given instead of chosen (their weights are
    still the plain scores): a comparison with a run in fewer bits takes that run's choices where a close call may have
    fallen the other way, so that it measures rounding and not the choice."""
    out = torch.zeros_like(h)
    scores = sigmoid(h @ w[p + "router"].T)
    for t in range(h.shape[0]):
        ids = choose(scores[t], mlp["router"]["top"]) if forced is None or t not in forced else forced[t]
        for e in ids:
            out[t] += expert(scores[t, e] * h[t:t + 1], w, f"{p}e{e}.", mlp["expert"]["limit"])[0]
    return out


# --------------------------------------------------------------------------- the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[List[torch.Tensor]] = None,
            forced: Optional[Dict[int, Dict[int, List[int]]]] = None) -> torch.Tensor:
    """Logits [T, V] of one whole sequence; ``layers_out`` collects the stream after every layer; ``forced``
    {layer: {position: expert ids}}: see ``experts_ff``."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][list(tokens)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        m = layer["mixer"]
        if layer["type"] == "attention":
            src = m.get("kv_from")
            y, kept[i] = attention_mixer(h, w, p + "mix.", m, None if src is None else kept[src])
        elif layer["type"] == "delta":
            y = delta_mixer(h, w, p + "mix.", m, eps)
        elif layer["type"] == "parallel":
            left, _ = attention_mixer(h, w, p + "mix.left.", m["left"])
            right = linear_mixer(h, w, p + "mix.right.", m["right"], eps)
            y = 0.5 * (rms_norm(left, w[p + "mix.left.out"], eps) + rms_norm(right, w[p + "mix.right.out"], eps))
        else:
            raise ValueError(f"layer type {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp is not None:
            if mlp["kind"] == "dense":
                y = y + dense_ff(h, w, p + "mlp.")
            else:
                y = y + experts_ff(h, w, p + "mlp.", mlp, None if forced is None else forced.get(i))
        x = x + cfg["residual_mult"] * y
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
