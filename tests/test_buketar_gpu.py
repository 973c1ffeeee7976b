"""The Buketar design on the GPU against the plain implementation (tests/plain_buketar.py): each mechanism alone at its
kernel's own interface, then the engine - the sum of the streams after every layer run, whole prompts, prompts against
token-by-token decoding, portions down to two tokens, unequal batches against each request alone, slots, pages and state
used again, far keys in prompts and in decoding, states with a long memory, long decoding - and greedy generation through
``Runner.generate``."""
import functools
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import buketar_configs as C
import plain_buketar as P
from gpu_helpers import BF16_REL_MAX, BF16_REL_MEAN, F32_REL, random_tokens

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
NAMES = list(C.CONFIGS)
DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("buketar")
    return {n: C.write_model(str(root / n), C.CONFIGS[n]) for n in NAMES}


@functools.lru_cache(maxsize=None)
def _plain(d):
    return P.load_model_dir(d)


_LOGITS = {}


def plain_logits(d, tokens, forced=None):
    cfg, w = _plain(d)
    if forced:
        return P.forward(cfg, w, list(tokens), forced=forced)
    key = (d, tuple(tokens))
    if key not in _LOGITS:
        _LOGITS[key] = P.forward(cfg, w, list(tokens))
    return _LOGITS[key]


class Choices:
    """While it is open around a bfloat16 run, it notes which experts every router of the run chose, by slot, layer run
    and position; ``of(slot)`` hands them to the plain implementation ({run: {position: ids}}), which then takes the
    run's choices: where two scores lie within rounding of one another the run may choose the other expert, which is
    no fault, and the comparison is to measure everything else.  (The routers' own choices are tested exactly in 32-bit
    and at the kernels' interface.)  A 32-bit run is left alone: ``of`` gives ``None``.  Single-token steps run
    uncaptured meanwhile, since a replayed graph calls no Python."""

    def __init__(self, r, dtype):
        self.r, self.on = r, dtype == "bfloat16"
        self.seen = {}

    def __enter__(self):
        if not self.on:
            return self
        from rustyllm_b200.models.decoder import DecoderModel
        from rustyllm_b200.parts.moe import MoEMLP
        schedule = self.r.model.spec.schedule
        runs = [k for k, i in enumerate(schedule) if isinstance(self.r.model.blocks[i].feed_forward, MoEMLP)]
        self.saved = (MoEMLP.route, DecoderModel.forward, self.r.engine.use_graphs)
        rec = self

        def forward(model, step, cache):
            rec.step, rec.at = (step.slot_of_token.tolist(), step.positions.tolist()), 0
            return rec.saved[1](model, step, cache)

        def route(part, xn):
            ids, weights = rec.saved[0](part, xn)
            run = runs[rec.at]
            rec.at += 1
            for row, sl, pos in zip(ids.tolist(), *rec.step):
                rec.seen.setdefault(sl, {}).setdefault(run, {})[pos] = row
            return ids, weights
        MoEMLP.route, DecoderModel.forward = route, forward
        self.r.engine.use_graphs = False
        return self

    def __exit__(self, *exc):
        if self.on:
            from rustyllm_b200.models.decoder import DecoderModel
            from rustyllm_b200.parts.moe import MoEMLP
            MoEMLP.route, DecoderModel.forward, self.r.engine.use_graphs = self.saved

    def of(self, slot):
        return self.seen.get(slot) if self.on else None


@functools.lru_cache(maxsize=None)
def runner(d, dtype, max_cache_tokens=64 * 40, max_batch=8):
    from rustyllm_b200 import Runner
    return Runner.from_path(d, dtype=dtype, max_cache_tokens=max_cache_tokens, max_batch=max_batch)[0]


def close(got, ref, dtype, cfg, what, forced=True):
    """32-bit: 3e-5 of a logit row's rms.  bfloat16: the bounds of gpu_helpers (derived for three pre-norm layers) grown
    with the square root of the layer runs, where the plain implementation took the run's expert choices (``Choices``);
    where it could not (``forced=False``: a subprocess) a router's close call may fall the other way once its input is
    rounded, so a fifth of the rows may differ by more."""
    got, ref = got.detach().to("cpu", F64), ref.detach().to("cpu", F64)
    assert got.shape == ref.shape, f"{what}: {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    err = (got - ref).abs() / ref.pow(2).mean(dim=-1, keepdim=True).sqrt().clamp_min(1e-30)
    rows = err.max(dim=-1).values
    if dtype == "float32":
        assert rows.max().item() <= F32_REL, f"{what}: {rows.max().item():.3e} (row {rows.argmax().item()})"
        return
    grow = 2.0 * math.sqrt(max(1.0, len(C.running_layers(cfg)) / 3.0))
    bound = BF16_REL_MAX * grow
    # the rows' errors have a long tail: where two large scores of a sharp attention row are nearly equal, the rounding
    # of q and k moves its weights by several per cent.  Up to 3 % of the rows (two in short requests) may exceed the
    # bound, none three times the bound (a lost key, a key too many, a lost state or another expert show as 0.5 and more)
    over = (rows > bound).double().sum().item()
    if not forced:
        assert over <= max(2.0, 0.2 * rows.numel()), f"{what}: {over:.0f} of {rows.numel()} rows above {bound:.3f} (worst {rows.max().item():.3e})"
        return
    assert over <= max(2.0, 0.03 * rows.numel()), f"{what}: {over:.0f} of {rows.numel()} rows above {bound:.3f} (worst {rows.max().item():.3e})"
    assert rows.max().item() <= 3.0 * bound, f"{what}: max {rows.max().item():.3e} (row {rows.argmax().item()})"
    assert err.mean().item() <= BF16_REL_MEAN * grow, f"{what}: mean {err.mean().item():.3e}"


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def tdt(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def rounded(x, dtype):
    """What the kernel is given: the float64 test data rounded to the run's storage type."""
    return x.to(tdt(dtype)).to(F64)


def tol(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == "float32" else dict(rtol=1.2e-2, atol=1.2e-2)


def f32(x):
    return x.float().to(DEV)


def state_area(slots, nbytes, pad=256):
    """A per-slot state as the cache hands it out: a column range of a wider area, zeroed."""
    area = torch.zeros((slots, pad + nbytes + pad), dtype=torch.uint8, device=DEV)
    return area, area[:, pad:pad + nbytes]


class Step:
    """The integers of a step for kernels that take them one by one: sequences (slot, start, count)."""

    def __init__(self, seqs):
        pos, slot, cu = [], [], [0]
        for s, start, n in seqs:
            pos += list(range(start, start + n))
            slot += [s] * n
            cu.append(cu[-1] + n)
        self.positions, self.slot_of_token, self.cu_seqlens = i32(pos), i32(slot), i32(cu)
        self.seq_slots = i32([s for s, _, _ in seqs])
        self.q_lens = [n for _, _, n in seqs]
        self.M = len(pos)


# =========================================================================== mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 8, 9, 17])
@pytest.mark.parametrize("d", [7, 50, 64, 324, 2048])
def test_streams_opened_joined_and_read(dtype, S, d):
    from rustyllm_b200 import kernels as K
    torch.manual_seed(100 * S + d)
    M, top = 6, 3
    x0, w, ls = torch.randn(M, d, dtype=F64).float(), 1.0 + 0.2 * torch.randn(d), torch.rand(d)
    coef, to, mix = torch.randn(S), torch.randn(S), torch.randn(S, S)
    t = dict(rtol=3e-5, atol=3e-5) if dtype == "float32" else dict(rtol=8e-3, atol=8e-3)
    X = torch.empty(M, S, d, device=DEV)
    out = torch.empty(M, d, dtype=tdt(dtype), device=DEV)
    K.streams_open(x0.to(DEV), X, coef.to(DEV), w.to(DEV), 1e-4, out)
    ref = torch.stack([x0.double()] * S)                                        # the plain implementation's [S, M, d]
    assert torch.equal(X.cpu(), torch.stack([x0] * S, dim=1))
    torch.testing.assert_close(out.cpu().double(), P.rms_norm(P.streams_read(ref, coef.double()), w.double(), 1e-4), **t)
    # a join from a dense y with a factor, streams that differ, and the next read
    ref = torch.randn(S, M, d, dtype=F64).float().double()
    X = ref.transpose(0, 1).float().contiguous().to(DEV)
    y = torch.randn(M, d)
    K.streams_join(X, y.to(DEV), mix.to(DEV), to.to(DEV), ls.to(DEV), y_factor=0.75, coef=coef.to(DEV), norm_weight=w.to(DEV), eps=1e-4, out=out)
    ref = P.streams_join(ref, 0.75 * y.double() * ls.double(), mix.double(), to.double())
    torch.testing.assert_close(X.cpu().double().transpose(0, 1), ref, rtol=1e-5, atol=1e-5 * S)
    torch.testing.assert_close(out.cpu().double(), P.rms_norm(P.streams_read(ref, coef.double()), w.double(), 1e-4), **t)
    # a join from experts' rows, nothing read
    ref = X.cpu().double().transpose(0, 1)
    rows, wts = torch.randn(40, d), torch.rand(M, top)
    row = torch.randperm(40)[:M * top].to(torch.int32)
    K.streams_join(X, rows.to(DEV), mix.to(DEV), to.to(DEV), None, row=row.to(DEV), weights=wts.to(DEV))
    yy = (rows.double()[row.long()].view(M, top, d) * wts.double().unsqueeze(2)).sum(1)
    ref = P.streams_join(ref, yy, mix.double(), to.double())
    torch.testing.assert_close(X.cpu().double().transpose(0, 1), ref, rtol=1e-5, atol=1e-5 * S)
    # the plain sum of some tokens' streams
    some = torch.empty(3, d, dtype=tdt(dtype), device=DEV)
    K.streams_read(X, None, w.to(DEV), 1e-6, some, i32([5, 0, 2]))
    torch.testing.assert_close(some.cpu().double(), P.rms_norm(X.cpu().double().sum(1), w.double(), 1e-6)[[5, 0, 2]], **t)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 8])
@pytest.mark.parametrize("parts,n", [(3, 16), (2, 7), (1, 130)])
def test_filter_in_parts_and_single_tokens(dtype, taps, parts, n):
    """Two sequences: one by portions and single tokens, one by single tokens from the first; the filter's output as
    parts of the channels; the step kernel against the two kernels it stands for."""
    from rustyllm_b200 import kernels as K
    torch.manual_seed(10 * taps + n)
    W = parts * n
    z = [rounded(torch.randn(t, W, dtype=F64), dtype) for t in (14, 9)]
    taps_w, bias = torch.randn(W, taps, dtype=F64).float(), torch.randn(W)
    area, state = state_area(3, 4 * max(taps - 1, 0) * W)
    plan = [[(2, 0, 3), (1, 0, 5)]] + [[(2, 3 + k, 1), (1, 5 + k, 1)] for k in range(4)] + [[(2, 7, 2)]] + [[(2, 9 + k, 1)] for k in range(5)]
    got = {2: torch.zeros(14, W, dtype=F64), 1: torch.zeros(9, W, dtype=F64)}
    src = {2: z[0], 1: z[1]}
    for seqs in plan:
        st = Step(seqs)
        wide = torch.zeros(st.M, W + 16, dtype=tdt(dtype), device=DEV)
        wide[:, 5:5 + W] = torch.cat([src[s][a:a + c] for s, a, c in seqs]).to(tdt(dtype)).to(DEV)
        x = wide[:, 5:5 + W]
        if all(c == 1 for _, _, c in seqs):
            out = torch.empty(st.M, W, dtype=tdt(dtype), device=DEV)
            K.short_conv_step(x, f32(taps_w), f32(bias), False, st.seq_slots, state, out)
            res = out.cpu().double()
        else:
            out = torch.empty(parts, st.M + 3, n, dtype=tdt(dtype), device=DEV)
            K.short_conv(x, f32(taps_w), f32(bias), False, st.slot_of_token, state, out)
            K.short_conv_state(x, taps, st.cu_seqlens, st.seq_slots, state)
            res = torch.cat([out[b, :st.M] for b in range(parts)], dim=1).cpu().double()
        o = 0
        for s, a, c in seqs:
            got[s][a:a + c] = res[o:o + c]
            o += c
    for s, t in ((2, 14), (1, 9)):
        torch.testing.assert_close(got[s], P.causal_filter(src[s], taps_w.double(), bias.double())[:t], **tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("parts,n", [(2, 96), (3, 16), (4, 7), (1, 40), (1, 300), (5, 8)])
@pytest.mark.parametrize("portions", [[(1, 1, 2, 1, 40, 1, 3), (30, 19)], [(300,), (33, 1, 32)], [(2, 2, 2, 1, 1), (270, 1)]])
def test_gated_recurrence_across_steps(dtype, parts, n, portions):
    """Two sequences, cut differently; spans of tokens and single tokens; decays from a memory of thousands of tokens to
    a few; the state is carried in the slot's state area."""
    from rustyllm_b200 import kernels as K
    torch.manual_seed(parts * 100 + n + len(portions[0]))
    W = parts * n
    T = [sum(p) for p in portions]
    mats_r, mats_i = (rounded(torch.randn(parts, n, n, dtype=F64) / math.sqrt(n), dtype) for _ in range(2))
    bias_r, bias_i = torch.randn(parts, n), torch.randn(parts, n)
    lam = -9.0 + 10.0 * torch.rand(W)
    u = [rounded(torch.randn(t, W, dtype=F64), dtype) for t in T]
    y = [rounded(torch.randn(t, W, dtype=F64), dtype) for t in T]
    w = torch.stack([mats_r, mats_i], dim=1).reshape(parts, 2 * n, n).to(tdt(dtype)).to(DEV)
    zb = torch.stack([bias_r, bias_i], dim=1).reshape(parts, 2 * n).to(DEV)
    area, state = state_area(3, 4 * W)
    slots, at = [1, 2], [0, 0]
    got = [torch.zeros(t, W, dtype=F64) for t in T]
    for k in range(max(len(p) for p in portions)):
        seqs = [(slots[b], at[b], portions[b][k]) for b in range(2) if k < len(portions[b])]
        st = Step(seqs)
        rows_u = torch.cat([u[slots.index(s)][a:a + c] for s, a, c in seqs])
        rows_y = torch.cat([y[slots.index(s)][a:a + c] for s, a, c in seqs]).to(tdt(dtype)).to(DEV)
        out = torch.empty(st.M, W, dtype=tdt(dtype), device=DEV)
        if all(c == 1 for _, _, c in seqs):
            K.gated_recurrence_step(rows_u.to(tdt(dtype)).to(DEV), w, zb, f32(lam), 8.0, rows_y, out, state, st.seq_slots)
        else:
            part_u = rows_u.view(st.M, parts, n).transpose(0, 1).contiguous()
            z = torch.cat([part_u @ mats_r.transpose(1, 2), part_u @ mats_i.transpose(1, 2)], dim=2)
            K.gated_recurrence(part_u.to(tdt(dtype)).to(DEV), f32(z), zb, f32(lam), 8.0, rows_y, out, state, st.cu_seqlens, st.seq_slots, st.q_lens)
        o = 0
        for s, a, c in seqs:
            got[slots.index(s)][a:a + c] = out[o:o + c].cpu().double()
            o += c
            at[slots.index(s)] += c
    for b in range(2):
        r, i = P.recurrence_gates(u[b], mats_r, bias_r.double()), P.recurrence_gates(u[b], mats_i, bias_i.double())
        S = P.gated_recurrence(u[b], r, i, lam.double())
        assert (torch.exp(-8.0 * r * P.softplus(lam.double())) > 0.999).any(), "no channel with a long memory"
        torch.testing.assert_close(got[b], S * P.gelu_tanh(y[b]), **(dict(rtol=3e-5, atol=1e-5) if dtype == "float32" else dict(rtol=1.2e-2, atol=1.2e-2)))
        torch.testing.assert_close(state[slots[b]].view(torch.float32).cpu().double(), S[-1], rtol=1e-4, atol=1e-5)


def test_a_decay_close_to_one_keeps_its_digits_over_thousands_of_tokens():
    """log a = -1e-4 or so, the same every token: a decay rounded to float would be off by the same amount 6,000 times."""
    from rustyllm_b200 import kernels as K
    torch.manual_seed(5)
    T, n = 6000, 8
    lam = torch.linspace(-13.0, -7.0, n)
    u, y = torch.ones(T, n, dtype=F64), torch.full((T, n), 3.0, dtype=F64)
    z = torch.zeros(1, T, 2 * n)
    for cut in ([6000], [1, 4000, 7, 1992]):
        area, state = state_area(1, 4 * n)
        at = 0
        for c in cut:
            st = Step([(0, at, c)])
            out = torch.empty(c, n, device=DEV)
            K.gated_recurrence(f32(u[at:at + c].view(1, c, n)), z[:, at:at + c].contiguous().to(DEV), torch.zeros(1, 2 * n, device=DEV), lam.to(DEV), 8.0, f32(y[at:at + c]), out, state,
                               st.cu_seqlens, st.seq_slots, st.q_lens)
            at += c
        half = torch.full((T, n), 0.5, dtype=F64)
        S = P.gated_recurrence(u, half, half, lam.double())
        torch.testing.assert_close(state[0].view(torch.float32).cpu().double(), S[-1], rtol=2e-6, atol=0.0)


@pytest.mark.parametrize("E,top", [(12, 3), (6, 6), (40, 2), (7, 1), (1, 1)])
@pytest.mark.parametrize("M", [5, 200])
@pytest.mark.parametrize("factor", [1.0, 2.5])
def test_router_with_sigmoid_scores_times_a_constant(E, top, M, factor):
    from rustyllm_b200 import kernels as K
    torch.manual_seed(E * 10 + top)
    d = 48
    x = torch.randn(M, d, dtype=F64).float()
    wr = (torch.randn(E, d, dtype=F64) * 1.5 / math.sqrt(d)).float()
    logits = x.double() @ wr.double().T
    ids = torch.empty(M, top, dtype=torch.int32, device=DEV)
    wts = torch.empty(M, top, dtype=torch.float32, device=DEV)
    for way in ("route", "select"):
        ids.zero_(), wts.zero_()
        if way == "route":
            K.moe_route_scored(x.to(DEV), wr.to(DEV), None, top, 1, 1, ids, wts, softmax_all=False, group_top=2, renorm=False, weight_scale=factor)
        else:
            K.moe_select_scored(logits.float().to(DEV), None, top, 1, 1, ids, wts, softmax_all=False, group_top=2, renorm=False, weight_scale=factor)
        for m in range(M):
            s = P.sigmoid(logits[m])
            want = sorted(range(E), key=lambda e: (-s[e].item(), e))[:top]
            order = sorted(s.tolist(), reverse=True)
            if E > 1 and min(order[i] - order[i + 1] for i in range(E - 1)) < 1e-6:
                continue                                   # a tie within float rounding
            assert ids[m].tolist() == want, f"{way} token {m}"
            torch.testing.assert_close(wts[m].cpu().double(), s[want] * factor, rtol=2e-5, atol=1e-7)


@pytest.mark.parametrize("dtype,grouped", [("float32", False), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("M,E,top,d,F", [(1, 4, 2, 64, 24), (7, 6, 3, 128, 40), (300, 5, 2, 64, 48), (900, 3, 3, 72, 136)])
def test_experts_with_the_clamped_gate(dtype, grouped, M, E, top, d, F):
    from rustyllm_b200 import kernels as K
    torch.manual_seed(M + F)
    limit, alpha = 0.8, 1.702
    x = rounded(torch.randn(M, d, dtype=F64), dtype)
    gate, up = (rounded(torch.randn(E, F, d, dtype=F64) / math.sqrt(d), dtype) for _ in range(2))
    down = rounded(torch.randn(E, d, F, dtype=F64) / math.sqrt(F), dtype)
    ids = torch.stack([torch.randperm(E)[:top] for _ in range(M)]).to(torch.int32)
    wts = torch.rand(M, top)
    want = torch.zeros(M, d, dtype=F64)
    for e in range(E):
        w = {"gate": gate[e], "up": up[e], "down": down[e]}
        y = P.clamped_expert(x, w, "", limit)
        for c in range(top):
            want += torch.where(ids[:, c:c + 1] == e, wts[:, c:c + 1].double() * y, torch.zeros_like(y))
    assert ((x @ gate[0].T) > limit).any() and ((x @ up[0].T) < -limit).any() and ((x @ up[0].T) > limit).any()
    xd, dd = x.to(tdt(dtype)).to(DEV), down.to(tdt(dtype)).to(DEV)
    turn = torch.stack([gate, up], dim=2).to(tdt(dtype)).to(DEV).contiguous()            # [E, F, 2, d]
    apart = torch.stack([gate, up], dim=1).to(tdt(dtype)).to(DEV).contiguous()           # [E, 2, F, d]
    res = torch.zeros(M, d, device=DEV)
    t = dict(rtol=3e-5, atol=3e-5) if dtype == "float32" else dict(rtol=1e-2, atol=1.5e-2)
    if grouped:
        K.moe_experts_grouped(xd, turn, dd, ids.to(DEV), wts.to(DEV), res, act=(limit, alpha))
        torch.testing.assert_close(res.cpu().double(), want, **t)
        rows, row = K.moe_experts_grouped(xd, turn, dd, ids.to(DEV), wts.to(DEV), None, act=(limit, alpha))
        got = (rows.cpu().double()[row.cpu().long()].view(M, top, d) * wts.double().unsqueeze(2)).sum(1)
        torch.testing.assert_close(got, want, **t)
        K.check_device_errors()
    else:
        K.moe_experts(xd, apart, dd, ids.to(DEV), wts.to(DEV), res, act=(limit, alpha))
        torch.testing.assert_close(res.cpu().double(), want, **t)
        res.zero_()
        K.moe_experts(xd, turn, dd, ids.to(DEV), wts.to(DEV), res, interleaved=True, act=(limit, alpha))
        torch.testing.assert_close(res.cpu().double(), want, **t)


@pytest.mark.parametrize("M", [3, 20, 64, 100, 200, 1500])
def test_clamped_gate_in_the_epilogue_of_the_tensor_core_product(M):
    """Every form of the product: few tokens with the K range in parts and whole, many tokens (persistent)."""
    from rustyllm_b200 import kernels as K
    torch.manual_seed(M)
    for d, I, limit in ((1024, 96, 0.7), (136, 320, 1.4)):
        x = torch.randn(M, d).to(torch.bfloat16)
        wg, wu = (torch.randn(I, d) / math.sqrt(d)).to(torch.bfloat16), (torch.randn(I, d) / math.sqrt(d)).to(torch.bfloat16)
        w = torch.stack([wg, wu], dim=1).reshape(2 * I, d).contiguous()
        out = torch.empty(M, I, dtype=torch.bfloat16, device=DEV)
        K.gemm_tc(x.to(DEV), w.to(DEV), out, K.OUT_CLAMPED, act=(limit, 1.702))
        K.check_device_errors()
        want = P.clamped_expert(x.double(), {"gate": wg.double(), "up": wu.double(), "down": torch.eye(I, dtype=F64)}, "", limit)
        torch.testing.assert_close(out.cpu().double(), want, rtol=1.2e-2, atol=1.2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,hd,rd,r,dims", [(3, 24, 8, 32, 8), (2, 10, 6, 20, 6), (4, 16, 16, 40, 8), (1, 7, 5, 11, 4), (5, 64, 32, 128, 32)])
@pytest.mark.parametrize("half", [True, False])
def test_latent_rows_and_query_parts_turned_with_a_magnitude(dtype, H, hd, rd, r, dims, half):
    """No query latent: the queries are columns of the same row; positions up to 5,000 in scattered pages."""
    from rustyllm_b200 import kernels as K
    torch.manual_seed(hd + r)
    positions = [0, 1, 63, 64, 65, 130, 4999]
    M, mag = len(positions), 1.37
    qc = H * (hd + rd)
    u = rounded(torch.randn(M, qc + r + rd + 3, dtype=F64), dtype)
    w = (1.0 + 0.2 * torch.randn(r)).float()
    pages = 80
    table = i32([torch.randperm(pages).tolist()])
    k_pool = torch.zeros(pages, 1, 64, r + rd, dtype=tdt(dtype), device=DEV)
    inv = torch.tensor([50.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32)
    ud = u.to(tdt(dtype)).to(DEV)
    K.latent_prepare(ud[:, qc:], 0, r, rd, None, f32(w), 1e-5, None, i32(positions), i32([0] * M), table, inv.to(DEV), dims, not half, k_pool,
                     magnitude=mag)
    out = torch.zeros(M, H * (r + rd), dtype=tdt(dtype), device=DEV)
    K.latent_query(ud[:, :qc], out, H, hd, rd, r, i32(positions), inv.to(DEV), dims, not half, magnitude=mag)

    def turned(x, p):
        y = x.clone()
        for i in range(dims // 2):
            a, b = (i, i + dims // 2) if half else (2 * i, 2 * i + 1)
            ang = float(np.float32(p) * np.float32(inv[i]))
            c, s = mag * math.cos(ang), mag * math.sin(ang)
            y[a], y[b] = x[a] * c - x[b] * s, x[b] * c + x[a] * s
        return y
    for m, p in enumerate(positions):
        want = torch.cat([P.rms_norm(u[m, qc:qc + r], w.double(), 1e-5), turned(u[m, qc + r:qc + r + rd], p)])
        got = k_pool[table[0, p // 64], 0, p % 64].cpu().double()
        torch.testing.assert_close(got, want, **tol(dtype))
        for h in range(H):
            q = u[m, h * (hd + rd) + hd:(h + 1) * (hd + rd)]
            torch.testing.assert_close(out[m, h * (r + rd) + r:(h + 1) * (r + rd)].cpu().double(), turned(q, p), **tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,H,N,K_", [(1, 3, 32, 24), (17, 16, 64, 128), (64, 4, 48, 96), (33, 2, 7, 5)])
def test_a_product_a_head_with_an_element_gate(dtype, M, H, N, K_):
    from rustyllm_b200 import kernels as K
    torch.manual_seed(M + N)
    x, w = rounded(torch.randn(M, H * K_, dtype=F64), dtype), rounded(torch.randn(H, N, K_, dtype=F64) / math.sqrt(K_), dtype)
    g = rounded(torch.randn(M, 5 + H * N, dtype=F64), dtype)
    out = torch.empty(M, H * N, dtype=tdt(dtype), device=DEV)
    K.heads_linear(x.to(tdt(dtype)).to(DEV), K_, w.to(tdt(dtype)).to(DEV), out, N, gate=g.to(tdt(dtype)).to(DEV)[:, 5:])
    want = torch.einsum("mhk,hnk->mhn", x.view(M, H, K_), w).reshape(M, H * N) * P.sigmoid(g[:, 5:])
    torch.testing.assert_close(out.cpu().double(), want, **tol(dtype))


# =========================================================================== the engine
@pytest.mark.parametrize("name", NAMES)
def test_sum_of_the_streams_after_every_layer_run(dirs, name):
    d = dirs[name]
    cfg, w = _plain(d)
    r = runner(d, "float32")
    toks = random_tokens(cfg["vocab"], 37, 5)
    want = []
    P.forward(cfg, w, toks, want)
    caps = []
    blocks = r.model.blocks
    for b in blocks:
        def wrapped(x, step, cache, *a, _f=b.forward, **k):
            out = _f(x, step, cache, *a, **k)
            caps.append(x.detach().sum(1).cpu().double())
            return out
        b.forward = wrapped
    try:
        s = r.engine.alloc_slot()
        r.engine.step([s], [toks], None)
        r.engine.free_slot(s)
    finally:
        for b in blocks:
            del b.forward
    assert len(caps) == len(want) == len(C.running_layers(cfg))
    for i, (got, ref) in enumerate(zip(caps, want)):
        scale = ref.pow(2).mean().sqrt().item()
        assert (got - ref).abs().max().item() <= 3e-5 * scale, f"{name}: the streams after layer run {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_first_tokens(dirs, name, dtype):
    d = dirs[name]
    cfg, _ = _plain(d)
    r = runner(d, dtype)
    for n, seed in ((1, 1), (2, 2), (65, 3), (130, 4)):
        toks = random_tokens(cfg["vocab"], n, seed)
        with Choices(r, dtype) as ch:
            s = r.engine.alloc_slot()
            got = r.engine.step([s], [toks], "all")
            r.engine.free_slot(s)
        close(got, plain_logits(d, toks, ch.of(s)), dtype, cfg, f"{name} {dtype} prompt of {n}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_token_by_token_equals_whole(dirs, name, dtype):
    """A prompt, then 70 single tokens (across a page's border); and 140 single tokens from the very first."""
    d = dirs[name]
    cfg, _ = _plain(d)
    r = runner(d, dtype)
    for n, first in ((120, 50), (140, 1)):
        toks = random_tokens(cfg["vocab"], n, 11 + n)
        with Choices(r, dtype) as ch:
            s = r.engine.alloc_slot()
            rows = [r.engine.step([s], [toks[:first]], "last")]
            for t in toks[first:]:
                rows.append(r.engine.step([s], [[t]], "last"))
            r.engine.free_slot(s)
        close(torch.cat(rows), plain_logits(d, toks, ch.of(s))[first - 1:], dtype, cfg, f"{name} {dtype} decode after {first}")
    if dtype == "bfloat16":
        # the captured single-token step (what generation replays) against the uncaptured one: the same kernels
        toks = random_tokens(cfg["vocab"], 40, 9)
        outs = []
        for graphs in (False, True):
            saved, r.engine.use_graphs = r.engine.use_graphs, graphs
            s = r.engine.alloc_slot()
            rows = [r.engine.step([s], [toks[:30]], "last")] + [r.engine.step([s], [[t]], "last") for t in toks[30:]]
            r.engine.free_slot(s)
            r.engine.use_graphs = saved
            outs.append(torch.cat(rows))
        assert torch.equal(outs[0], outs[1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_prompt_then_decoding(dirs, name, dtype):
    """700 tokens at once, then single tokens: far keys and an old state."""
    d = dirs[name]
    cfg, _ = _plain(d)
    r = runner(d, dtype)
    toks = random_tokens(cfg["vocab"], 730, 21)
    with Choices(r, dtype) as ch:
        s = r.engine.alloc_slot()
        rows = [r.engine.step([s], [toks[:700]], [[0, 350, 699]])]
        for t in toks[700:]:
            rows.append(r.engine.step([s], [[t]], "last"))
        r.engine.free_slot(s)
    ref = plain_logits(d, toks, ch.of(s))
    close(torch.cat(rows), ref[[0, 350] + list(range(699, 730))], dtype, cfg, f"{name} {dtype} long prompt")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,r,rd", [(4, 40, 24), (2, 22, 6), (20, 64, 32)])
def test_a_far_key_that_stands_out_decides_the_output(tmp_path, dtype, H, r, rd):
    """One latent layer whose queries look for one token: W_q maps the marked token's input onto the query that meets
    its own key far above all others, so the position of its latest occurrences decides the row.  The marked token stands
    at a page's last and first place and hundreds of positions back; seen from a prompt, a portion and single tokens."""
    d, V, dk, dv, n = 96, 40, 8, 12, 520
    cfg = {"architecture": "Buketar", "vocab": V, "width": d, "norm": {"eps": 1e-5}, "streams": 2,
           "layers": [C.latent(H, dk, rd, dv, r, 0.2, None, base=1.0e4, scaling=(4.0, 64, 16.0, 1.0))]}
    w = C.draw_weights(cfg, 7)
    g = torch.Generator().manual_seed(3)
    # a row of the embedding of its own for the marked token 0 (orthogonal to the rest), one direction of the latent it
    # alone fills, one of the plain key part that this direction feeds, and queries along it whatever the asking token
    e0 = torch.zeros(d, dtype=F64)
    e0[0] = 1.0
    emb = torch.randn(V, d, generator=g, dtype=F64)
    emb[:, 0] = 0.0
    emb[:, 1] = 3.0                                          # every token carries a constant in channel 1
    emb[0] = e0 * 6.0
    emb[0, 1] = 3.0
    down = w["l0.mix.dkv"].double()
    down[0] = e0 * 4.0                                       # latent direction 0: the marked token alone
    uk = w["l0.mix.uk"].double().view(H, dk, r)
    uk[:, 0] = 0.0
    uk[:, 0, 0] = 3.0
    q = w["l0.mix.q"].double().view(H, dk + rd, d)
    q[:, 0] = 0.0
    q[:, 0, 1] = 8.0
    w.update({"embed": emb.to(torch.bfloat16), "l0.mix.dkv": down.to(torch.bfloat16), "l0.mix.uk": uk.reshape(H * dk, r).to(torch.bfloat16),
              "l0.mix.q": q.reshape(H * (dk + rd), d).to(torch.bfloat16), "l0.mix.dkv.norm": torch.ones(r, dtype=torch.bfloat16)})
    path = C.write_model(str(tmp_path / "m"), cfg, weights=w)
    pc, pw = P.load_model_dir(path)
    run = runner(path, dtype)
    for far in (0, 63, 64, 127, 5):
        toks = [t % (V - 1) + 1 for t in random_tokens(V, n, far)]
        toks[far] = 0
        ref = P.forward(pc, pw, toks)
        other = list(toks)
        other[far] = 1
        moved = (P.forward(pc, pw, other)[-40:] - ref[-40:]).abs().max(dim=-1).values / ref[-40:].pow(2).mean(-1).sqrt()
        assert moved.min() > 0.3, "the far token does not show in every late row"
        s = run.engine.alloc_slot()
        rows = [run.engine.step([s], [toks[:480]], [[479]]), run.engine.step([s], [toks[480:500]], "all")]
        rows += [run.engine.step([s], [[t]], "last") for t in toks[500:]]
        run.engine.free_slot(s)
        close(torch.cat(rows), ref[479:], dtype, cfg, f"far key at {far}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("size", [2, 3, 7, 64, 100])
def test_prompt_in_portions(dirs, name, dtype, size):
    d = dirs[name]
    cfg, _ = _plain(d)
    r = runner(d, dtype)
    toks = random_tokens(cfg["vocab"], 140, 31)
    with Choices(r, dtype) as ch:
        s = r.engine.alloc_slot()
        rows = [r.engine.step([s], [toks[a:a + size]], "all") for a in range(0, len(toks), size)]
        r.engine.free_slot(s)
    close(torch.cat(rows), plain_logits(d, toks, ch.of(s)), dtype, cfg, f"{name} {dtype} portions of {size}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_reuse_slots_and_pages(dirs, name, dtype):
    """Two batches of unequal requests, one after the other, through a cache that only just holds one: every slot,
    page and state is used again; each request must come out as it does alone."""
    from rustyllm_b200 import Runner
    d = dirs[name]
    cfg, _ = _plain(d)
    r = Runner.from_path(d, dtype=dtype, max_cache_tokens=64 * 7, max_batch=3)[0]
    for batch in range(2):
        lens = [(1, 130, 67), (70, 3, 129)][batch]
        reqs = [random_tokens(cfg["vocab"], n + 12, 100 * batch + n) for n in lens]
        with Choices(r, dtype) as ch:
            slots = [r.engine.alloc_slot() for _ in reqs]
            got = [[] for _ in reqs]
            out = r.engine.step(slots, [q[:n] for q, n in zip(reqs, lens)], "last")
            for b in range(3):
                got[b].append(out[b:b + 1])
            live = list(range(3))
            for k in range(12):
                if k == 6:                                        # the first request ends early; its slot is given back
                    gone = live.pop(0)
                    r.engine.free_slot(slots[gone])
                out = r.engine.step([slots[b] for b in live], [[reqs[b][lens[b] + k]] for b in live], "last")
                for j, b in enumerate(live):
                    got[b].append(out[j:j + 1])
            for b in live:
                r.engine.free_slot(slots[b])
        for b, q in enumerate(reqs):
            rows = torch.cat(got[b])
            ref = plain_logits(d, q[:lens[b] - 1 + rows.shape[0]], ch.of(slots[b]))[lens[b] - 1:lens[b] - 1 + rows.shape[0]]
            close(rows, ref, dtype, cfg, f"{name} {dtype} batch {batch} request {b}")
    r.cache.check()


@pytest.mark.parametrize("name", NAMES)
def test_logits_do_not_depend_on_the_batch_or_the_cut_in_32_bit(dirs, name):
    d = dirs[name]
    cfg, _ = _plain(d)
    r = runner(d, "float32")
    toks, beside = random_tokens(cfg["vocab"], 90, 5), random_tokens(cfg["vocab"], 33, 6)

    def alone(cuts):
        s = r.engine.alloc_slot()
        rows, at = [], 0
        for c in cuts:
            rows.append(r.engine.step([s], [toks[at:at + c]], "all"))
            at += c
        r.engine.free_slot(s)
        return torch.cat(rows)
    whole = alone([90])
    s = [r.engine.alloc_slot() for _ in range(2)]
    both = r.engine.step(s, [beside, toks], "all")[33:]
    for x in s:
        r.engine.free_slot(x)
    scale = whole.pow(2).mean().sqrt().item()
    for what, got in (("batch", both), ("cut", alone([2, 30, 1, 1, 56])), ("tokens", alone([1] * 90))):
        assert (got - whole).abs().max().item() <= 2e-5 * scale, f"{name}: {what}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_in_one_step(dirs, dtype):
    """70 sequences of 1 to 60 tokens in one prompt step and in single-token steps: more than the few-token forms of the
    kernels take (in both dtypes a batch of more than 64), each against the plain implementation."""
    from rustyllm_b200 import Runner
    d = dirs["C"]
    cfg, _ = _plain(d)
    r = Runner.from_path(d, dtype=dtype, max_cache_tokens=64 * 80, max_batch=70)[0]
    lens = [1 + (i * 17) % 60 for i in range(70)]
    reqs = [random_tokens(cfg["vocab"], n + 3, i) for i, n in enumerate(lens)]
    with Choices(r, dtype) as ch:
        slots = [r.engine.alloc_slot() for _ in reqs]
        outs = [r.engine.step(slots, [q[:n] for q, n in zip(reqs, lens)], "last")]
        for k in range(3):
            outs.append(r.engine.step(slots, [[q[n + k]] for q, n in zip(reqs, lens)], "last"))
    for b in range(0, 70, 3):
        ref = plain_logits(d, reqs[b], ch.of(slots[b]))[lens[b] - 1:]
        close(torch.stack([o[b] for o in outs]), ref, dtype, cfg, f"{dtype} sequence {b} of 70")


@pytest.mark.parametrize("seed", range(12))
@pytest.mark.parametrize("dtype", DTYPES)
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    from rustyllm_b200 import Runner
    cfg = C.random_config(seed)
    d = C.write_model(str(tmp_path / "m"), cfg, seed=seed)
    r = Runner.from_path(d, dtype=dtype, max_cache_tokens=64 * 12, max_batch=4)[0]
    a, b = random_tokens(cfg["vocab"], 80, seed), random_tokens(cfg["vocab"], 21, seed + 50)
    with Choices(r, dtype) as ch:
        s = [r.engine.alloc_slot(), r.engine.alloc_slot()]
        rows_a = [r.engine.step([s[0]], [a[:40]], "all")]
        out = r.engine.step(s, [a[40:75], b[:20]], "all")                 # a portion beside a fresh prompt
        rows_a.append(out[:35])
        rows_b = [out[35:]]
        for k in range(5):
            rows_a.append(r.engine.step([s[0]], [[a[75 + k]]], "last"))
        rows_b.append(r.engine.step([s[1]], [[b[20]]], "last"))
    close(torch.cat(rows_a), plain_logits(d, a, ch.of(s[0])), dtype, cfg, f"random {seed} {dtype} a")
    close(torch.cat(rows_b), plain_logits(d, b, ch.of(s[1])), dtype, cfg, f"random {seed} {dtype} b")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_runner(dirs, name, dtype):
    from rustyllm_b200 import GenerationOptions, SamplerConfig
    d = dirs[name]
    cfg, w = _plain(d)
    r = runner(d, dtype)
    prompts = [random_tokens(cfg["vocab"], n, 60 + n) for n in (3, 70, 20)]
    new = 24
    results = r.generate(prompts, GenerationOptions(max_tokens=new, sampler=SamplerConfig.greedy(), ignore_eos=True))
    again = r.generate(prompts, GenerationOptions(max_tokens=new, sampler=SamplerConfig.greedy(), ignore_eos=True, prefill_step_tokens=16))
    for p, got, cut in zip(prompts, results, again):
        tokens = list(got.token_ids)
        assert len(tokens) == new
        # follow the framework's own tokens and require that each is the plain implementation's best, or within
        # rounding of it (bfloat16 may pick the other of two near-equal logits, or another expert at a close call)
        ref = plain_logits(d, p + tokens[:-1])[len(p) - 1:]
        behind = [(ref[i].max() - ref[i, t]).item() / ref[i].std().item() for i, t in enumerate(tokens)]
        if dtype == "float32":
            assert max(behind) <= 1e-3, f"{name} request of {len(p)}: {max(behind)}"
            assert list(cut.token_ids) == tokens                   # the prompt in portions of 16: the same tokens
        else:
            assert sorted(behind)[-3] <= 0.25, f"{name} request of {len(p)}: {sorted(behind)[-4:]}"


def test_trace_replay_and_command_line(dirs, tmp_path):
    toks = random_tokens(C.CONFIGS["C"]["vocab"], 90, 77)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:80], "want": [0, 79]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[80:81], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[81:], "want": [8]}], "end": ["a"]}]
    d = dirs["C"]
    for dtype in DTYPES:
        cfg, _ = _plain(d)
        out = tmp_path / dtype
        p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert not (out / "1.f32").exists()
        ref = plain_logits(d, toks)
        got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1))
        got2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(1, -1))
        close(torch.cat([got0, got2]), ref[[0, 79, 89]], dtype, cfg, f"trace {dtype}", forced=False)
    exe = [sys.executable, os.path.join(root, "bin", "rustyllm"), d]
    p = subprocess.run(exe + ["--inspect"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0 and "Buketar" in p.stdout and "supported" in p.stdout, p.stderr[-2000:]
    for layer, row in (("0", "mixer_in.fused"), ("1", "ffn_router")):      # a recurrent layer; a latent layer
        p = subprocess.run(exe + ["--kernel-bench", "--kernel-bench-runs", "2", "--kernel-bench-layer", layer], capture_output=True, text=True,
                           timeout=600)
        assert p.returncode == 0 and row in p.stdout and "output" in p.stdout, (p.stdout[-2000:], p.stderr[-2000:])
    p = subprocess.run(exe + ["--prompt", "1 2 3", "--max-tokens", "5", "--temp", "0"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    p = subprocess.run(exe[:2] + [os.path.join(d, "config.json"), "--random", "--bench-json", "--batch", "2", "--prompt-len-range", "8,40",
                                  "--max-tokens", "6", "--context", "128", "--ignore-eos"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
