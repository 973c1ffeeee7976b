"""The Tigutar configuration, its description as parts and the plain implementation's own mechanisms (no GPU)."""
import copy
import math

import pytest
import torch

import plain_tigutar as P
import tigutar_configs as C
from rustyllm_b200 import ConfigError, resolve_architecture
from rustyllm_b200.cache.sequence_cache import KVNeed
from rustyllm_b200.config.tigutar import TigutarConfig
from rustyllm_b200.models.decoder import DecoderModel
from rustyllm_b200.parts import Runtime
from rustyllm_b200.parts.base import LayerNormRequest
from rustyllm_b200.weights.loader import check_checkpoint
from rustyllm_b200.weights.safetensors_io import Checkpoint

F64 = torch.float64


@pytest.mark.parametrize("name", list(C.CONFIGS) + list(range(12)))
def test_configuration_round_trip_and_tensor_names(tmp_path, name):
    cfg, rank = (C.CONFIGS[name], C.DECAY_RANK[name]) if isinstance(name, str) else C.random_config(name)
    arch = resolve_architecture(cfg)
    d = C.write_model(str(name), str(tmp_path / "m"), seed=1, cfg=cfg, rank=rank)
    ck = Checkpoint(d)
    typed = arch.parse_for(cfg, {n: tuple(e.shape) for n, e in ck.entries.items()})
    assert isinstance(typed, TigutarConfig) and arch.parse_config(typed.to_dict()) == typed
    spec = arch.build_spec(typed)
    model = DecoderModel(spec, Runtime(torch.device("cpu"), torch.float32))
    check_checkpoint(model.param_specs(), ck.entries, spec.ignored_tensors, d)     # every tensor named, none left over
    assert spec.ignored_tensors == ()
    # cache entries: one a layer that owns one; a layer on another's keys reads that one's
    entry_of, entries = {}, iter(range(len(cfg["layers"])))
    for i, (layer, (entry, writes)) in enumerate(zip(cfg["layers"], model.run_entry)):
        m = layer["mixer"]
        if m.get("kv_from") is not None:
            assert not writes and entry == entry_of[m["kv_from"]]
            continue
        assert writes and entry == next(entries)
        entry_of[i] = entry
        kv, state = model.entry_needs[entry]
        if layer["type"] == "attention":
            assert kv == KVNeed(m["kv_heads"], m["dim"], None, m["vdim"]) and state is None
        elif layer["type"] == "delta":
            assert kv is None
            kept = 4 * (m["conv"] - 1) * (2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"])
            assert state.nbytes >= kept + 4 * m["heads"] * m["dim"] * m["vdim"]
        else:
            a, r = m["left"], m["right"]
            assert kv == KVNeed(a["kv_heads"], a["dim"], (a.get("mask") or {}).get("size"), a["vdim"])
            assert state.nbytes == 4 * r["heads"] * r["dim"] * r["vdim"]


def test_the_decay_width_comes_from_the_checkpoint_or_from_its_own_key():
    cfg = C.CONFIGS["A"]
    arch = resolve_architecture(cfg)
    with pytest.raises(ConfigError, match="decay"):
        arch.build_spec(arch.parse_config(cfg))
    named = copy.deepcopy(cfg)
    named["layers"][2]["mixer"]["right"]["decay_rank"] = 7
    assert arch.parse_config(named).layers[2].mixer.right.decay_rank == 7
    arch.build_spec(arch.parse_config(named))
    assert arch.parse_for(cfg, {"l2.mix.right.a1": (9, 72)}).layers[2].mixer.right.decay_rank == 9


def test_configuration_errors_name_the_key():
    base = C.CONFIGS["A"]

    def broken(change):
        cfg = copy.deepcopy(base)
        change(cfg)
        return cfg
    cases = [
        (lambda c: c["layers"][0].__setitem__("type", "lightning"), "mixer type"),
        (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
        (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
        (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 7), "top"),
        (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
        (lambda c: c["layers"][0]["mlp"]["expert"].__setitem__("limit", 0), "limit"),
        (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 7), "dims"),
        (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 18), "rot"),
        (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "sparse"), "kind"),
        (lambda c: c["layers"][2]["mixer"]["right"].pop("tau"), "tau"),
        (lambda c: c["layers"][2]["mixer"]["right"].__setitem__("tau", -1.0), "tau"),
        (lambda c: c["layers"][2]["mixer"]["left"].__setitem__("kv_from", 1), "kv_from"),
        (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 0), "kv_from"),          # a delta layer has no keys
        (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 3), "kv_from"),
        (lambda c: c["layers"][3]["mixer"].__setitem__("vdim", 16), "kv_from"),
        (lambda c: c["layers"][3]["mixer"]["rot"].__setitem__("base", 5.0), "rotation"),
        (lambda c: c["layers"][1]["mixer"].__setitem__("mask", {"size": 9}), "window"),
        (lambda c: c.pop("norm"), "norm"),
        (lambda c: c.pop("residual_mult"), "residual_mult"),
    ]
    for change, word in cases:
        with pytest.raises(ConfigError, match=word):
            TigutarConfig.from_dict(broken(change))


def test_a_norm_request_goes_only_to_a_block_that_can_start_it():
    """Blocks say which kinds of norm they can start for the block behind them."""
    from rustyllm_b200.parts.base import NormRequest
    from rustyllm_b200.parts.block import ParallelSharedNormBlock, PreNormBlock
    from rustyllm_b200.parts.streams import HyperConnectedBlock, StreamRead
    w = torch.ones(4)
    asks = {"layer": LayerNormRequest(w, None, 1e-5), "rms": NormRequest(w, 1e-5), "streams": StreamRead(None, w, 1e-5)}
    takes = {"layer": ParallelSharedNormBlock, "rms": PreNormBlock, "streams": HyperConnectedBlock}
    for a, request in asks.items():
        for b, block in takes.items():
            assert isinstance(request, block.norm_requests) == (a == b)


# --------------------------------------------------------------------------- the plain implementation's mechanisms
def test_plain_layer_norm_has_a_bias():
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=F64)
    w, b = torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=F64), torch.tensor([0.0, 1.0, -1.0, 0.5], dtype=F64)
    torch.testing.assert_close(P.layer_norm(x, w, b, 0.0), (x - 3.0) / math.sqrt(3.5) * w + b)
    torch.testing.assert_close(P.layer_norm(torch.zeros(1, 4, dtype=F64), w, b, 1e-6), b.view(1, 4))


def test_plain_rotation_pairs_halves_and_leaves_the_rest():
    x = torch.arange(1.0, 9.0, dtype=F64).view(1, 1, 8).repeat(3, 1, 1)
    y = P.rotate_halves(x, [0, 1, 5], 4, 100.0)
    torch.testing.assert_close(y[0], x[0])                          # position 0: no turn
    torch.testing.assert_close(y[:, :, 4:], x[:, :, 4:])
    a0, a1 = 5 * 1.0, 5 * 100.0 ** (-2.0 / 4)
    want = [1 * math.cos(a0) - 3 * math.sin(a0), 2 * math.cos(a1) - 4 * math.sin(a1),
            3 * math.cos(a0) + 1 * math.sin(a0), 4 * math.cos(a1) + 2 * math.sin(a1)]
    torch.testing.assert_close(y[2, 0, :4], torch.tensor(want, dtype=F64))


def test_plain_attention_window_and_sink():
    T = 4
    q = torch.zeros((T, 1, 2), dtype=F64)                           # every score 0: plain means of what is seen
    k = torch.randn((T, 1, 2), dtype=F64)
    v = torch.tensor([1.0, 10.0, 100.0, 1000.0], dtype=F64).view(T, 1, 1)
    got = P.softmax_attention(q, k, v, 1.0, window=2).flatten()
    torch.testing.assert_close(got, torch.tensor([1.0, 5.5, 55.0, 550.0], dtype=F64))
    got = P.softmax_attention(q, k, v, 1.0, sink=torch.tensor([math.log(3.0)], dtype=F64)).flatten()   # three keys' worth without a value
    torch.testing.assert_close(got, torch.tensor([1 / 4, 11 / 5, 111 / 6, 1111 / 7], dtype=F64))


def test_plain_filter_reads_the_past_with_its_last_tap_on_the_present():
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    got = P.causal_filter(u, torch.tensor([[2.0, 3.0, 5.0]], dtype=F64)).flatten()
    torch.testing.assert_close(got, torch.tensor([5.0, 53.0, 532.0], dtype=F64))


def test_plain_delta_rule_replaces_what_a_key_holds():
    """With step size 1 and no decay, a unit key's value is replaced; the read-out sees the current token's write."""
    k = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 0.0]], dtype=F64)
    v = torch.tensor([[5.0], [7.0], [2.0]], dtype=F64)
    one = torch.ones(3, dtype=F64)
    o, S = P.delta_scan(k, k, v, one, one)
    torch.testing.assert_close(o.flatten(), torch.tensor([5.0, 7.0, 2.0], dtype=F64))
    torch.testing.assert_close(S, torch.tensor([[2.0], [7.0]], dtype=F64))
    o, S = P.delta_scan(k, k, v, 0.5 * one, 0.5 * one)               # decay first, then half of what is missing
    torch.testing.assert_close(o.flatten(), torch.tensor([2.5, 3.5, 0.625 + 0.5 * (2.0 - 0.625)], dtype=F64))
    torch.testing.assert_close(S[1], torch.tensor([1.75], dtype=F64))


def test_plain_linear_attention_decays_rows_and_reads_the_current_write():
    q = torch.ones((2, 2), dtype=F64)
    k = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64)
    v = torch.tensor([[1.0], [10.0]], dtype=F64)
    a = torch.tensor([[0.9, 0.9], [0.5, 0.25]], dtype=F64)
    o, S = P.linear_scan(q, k, v, a)
    torch.testing.assert_close(S, torch.tensor([[30.5], [40.5]], dtype=F64))
    torch.testing.assert_close(o.flatten(), torch.tensor([3.0, 71.0], dtype=F64))


def test_plain_experts_weigh_their_input():
    w = {"p.router": torch.tensor([[0.0], [1.0]], dtype=F64)}
    for e in range(2):
        w.update({f"p.e{e}.gate": torch.tensor([[2.0]], dtype=F64), f"p.e{e}.up": torch.tensor([[-9.0]], dtype=F64),
                  f"p.e{e}.down": torch.tensor([[1.0 + e]], dtype=F64)})
    h = torch.tensor([[1.0]], dtype=F64)
    mlp = {"router": {"top": 2}, "expert": {"limit": 1.25}}
    want = 0.0
    for e, z in ((0, 0.0), (1, 1.0)):
        s = 1 / (1 + math.exp(-z))
        g, u = min(2.0 * s, 1.25), max(-9.0 * s, -1.25)
        want += (1.0 + e) * g / (1 + math.exp(-1.702 * g)) * (u + 1.0)
    torch.testing.assert_close(P.experts_ff(h, w, "p.", mlp), torch.tensor([[want]], dtype=F64))
    assert P.choose(torch.tensor([0.2, 0.5, 0.5, 0.1], dtype=F64), 2) == [1, 2]      # ties go to the lower index
