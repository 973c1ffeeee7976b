"""The Buketar configuration, its description as parts and the plain implementation's own mechanisms (no GPU)."""
import copy
import math

import pytest
import torch

import buketar_configs as C
import plain_buketar as P
from rustyllm_b200 import ConfigError, resolve_architecture
from rustyllm_b200.cache.sequence_cache import KVNeed
from rustyllm_b200.config.buketar import BuketarConfig
from rustyllm_b200.config.spec import PartSpec
from rustyllm_b200.models.decoder import DecoderModel
from rustyllm_b200.parts import Runtime
from rustyllm_b200.parts.rope import YarnRotaryEmbedding
from rustyllm_b200.weights.loader import WeightsError, check_checkpoint, load_parameters
from rustyllm_b200.weights.safetensors_io import Checkpoint

F64 = torch.float64
CPU = Runtime(torch.device("cpu"), torch.float32)


@pytest.mark.parametrize("name", list(C.CONFIGS) + list(range(16)))
def test_configuration_round_trip_tensor_names_and_cache_entries(tmp_path, name):
    cfg = C.CONFIGS[name] if isinstance(name, str) else C.random_config(name)
    arch = resolve_architecture(cfg)
    typed = arch.parse_config(cfg)
    assert isinstance(typed, BuketarConfig) and arch.parse_config(typed.to_dict()) == typed
    spec = arch.build_spec(typed)
    model = DecoderModel(spec, CPU)
    ck = Checkpoint(C.write_model(str(tmp_path / "m"), cfg, seed=1))
    check_checkpoint(model.param_specs(), ck.entries, spec.ignored_tensors, "m")      # every tensor named, none left over
    model.bind(load_parameters(model.param_specs(), ck, torch.float32, torch.device("cpu"), spec.ignored_tensors))
    runs = C.running_layers(cfg)
    assert list(spec.schedule) == runs == P.running_order(cfg)
    # every run of a layer has an entry of its own
    assert len(model.entry_needs) == len(runs) and [e for e, w in model.run_entry if w] == list(range(len(runs)))
    for i, (kv, state) in zip(runs, model.entry_needs):
        m = cfg["layers"][i]["mixer"]
        if cfg["layers"][i]["type"] == "rglru":
            assert kv is None and state.nbytes >= 4 * m["width"] * m["conv"]
        else:
            assert kv == KVNeed(1, m["kv_rank"] + m["rot_dim"], None, 0) and state is None


def test_tensors_of_an_absent_feed_forward_may_be_in_the_file_and_others_may_not(tmp_path):
    cfg = C.CONFIGS["B"]
    weights = C.draw_weights(cfg, 0)
    weights["l1.norm2"] = weights["l1.norm1"]
    weights["l1.hc2.mix"] = weights["l1.hc1.mix"]
    arch = resolve_architecture(cfg)
    spec = arch.build_spec(arch.parse_config(cfg))
    model = DecoderModel(spec, CPU)
    ck = Checkpoint(C.write_model(str(tmp_path / "a"), cfg, weights=weights))
    check_checkpoint(model.param_specs(), ck.entries, spec.ignored_tensors, "a")
    weights["l1.hc3.mix"] = weights["l1.hc1.mix"]
    del weights["l2.mix.lam"]
    ck = Checkpoint(C.write_model(str(tmp_path / "b"), cfg, weights=weights))
    with pytest.raises(WeightsError, match="l2.mix.lam") as e:
        check_checkpoint(model.param_specs(), ck.entries, spec.ignored_tensors, "b")
    assert "l1.hc3.mix" in str(e.value)


def test_configuration_errors_name_the_key():
    base = C.CONFIGS["A"]
    cases = [
        (lambda c: c["layers"][0].__setitem__("type", "attention"), "mixer type"),
        (lambda c: c["layers"][0]["mixer"].__setitem__("blocks", 5), "blocks"),
        (lambda c: c["layers"][0]["mixer"].__setitem__("conv", 9), "taps"),
        (lambda c: c["layers"][0]["mixer"].pop("width"), "width"),
        (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 7), "top"),
        (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
        (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "kind"),
        (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
        (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 7), "dims"),
        (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 10), "rot_dim"),
        (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
        (lambda c: c.pop("streams"), "streams"),
        (lambda c: c["loop"].__setitem__("stop", 5), "loop"),
        (lambda c: c["loop"].__setitem__("stop", 1), "loop"),
        (lambda c: c.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    ]
    for change, word in cases:
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(ConfigError, match=word):
            BuketarConfig.from_dict(cfg)
    for key in ("loop", "logit_softcap"):
        cfg = copy.deepcopy(base)
        cfg[key] = None
        assert getattr(BuketarConfig.from_dict(cfg), key) is None


def test_a_block_of_streams_and_its_model_must_agree():
    arch = resolve_architecture(C.CONFIGS["A"])
    spec = arch.build_spec(arch.parse_config(C.CONFIGS["A"]))
    import dataclasses
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(dataclasses.replace(spec, streams=2), CPU)
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(dataclasses.replace(spec, streams=0), CPU)


@pytest.mark.parametrize("n,base,scaling", [(16, 1.0e5, (16.0, 128, 16.0, 2.0)), (8, 500.0, (8.0, 64, 8.0, 1.0)), (2, 100.0, (4.0, 32, 32.0, 1.0)),
                                            (64, 10000.0, (40.0, 4096, 32.0, 1.0)), (12, 30.0, None), (16, 10.0, (4.0, 8, 1.0, 1.0))])
def test_frequencies_and_magnitude_equal_the_plain_ones(n, base, scaling):
    rot = {"dims": n, "base": base}
    params = {"head_dim": n, "rotary_dim": n, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
        params.update(rot["scaling"])
    e = YarnRotaryEmbedding(CPU, **params)
    torch.testing.assert_close(e.inv_freq.double(), torch.tensor(P.frequencies(rot), dtype=F64), rtol=1e-6, atol=0.0)
    assert math.isclose(e.magnitude, P.magnitude(rot)) and not e.interleaved


# --------------------------------------------------------------------------- the plain implementation's mechanisms
def test_plain_streams_by_hand():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=F64)                 # two streams, one token, two columns
    torch.testing.assert_close(P.streams_read(X, torch.tensor([2.0, 0.5], dtype=F64)), torch.tensor([[7.0, 14.0]], dtype=F64))
    mix = torch.tensor([[1.0, 3.0], [0.0, 2.0]], dtype=F64)                     # stream 0 flows into both, stream 1 into itself
    y = torch.tensor([[100.0, 0.0]], dtype=F64)
    out = P.streams_join(X, y, mix, torch.tensor([1.0, -1.0], dtype=F64))
    torch.testing.assert_close(out, torch.tensor([[[101.0, 2.0]], [[3.0 + 20.0 - 100.0, 6.0 + 40.0]]], dtype=F64))


def test_plain_filter_and_recurrence_by_hand():
    z = torch.tensor([[1.0], [2.0], [4.0]], dtype=F64)
    y = P.causal_filter(z, torch.tensor([[10.0, 1.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    torch.testing.assert_close(y, torch.tensor([[1.5], [12.5], [24.5]], dtype=F64))
    lam = torch.tensor([math.log(math.e - 1.0)], dtype=F64)                      # softplus = 1
    r = torch.full((2, 1), 0.125, dtype=F64)                                     # log a = -1
    i = torch.full((2, 1), 0.5, dtype=F64)
    S = P.gated_recurrence(torch.tensor([[2.0], [6.0]], dtype=F64), r, i, lam)
    f = math.sqrt(1.0 - math.exp(-2.0))
    torch.testing.assert_close(S, torch.tensor([[f], [math.exp(-1.0) * f + 3.0 * f]], dtype=F64))


def test_plain_gates_take_their_own_part_of_the_channels():
    u = torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=F64)
    mats = torch.zeros(2, 2, 2, dtype=F64)
    mats[0, 0, 1], mats[1, 1, 0] = 1.0, -1.0                                     # out 0 reads in 1; out 3 reads in 2
    g = P.recurrence_gates(u, mats, torch.tensor([[0.0, 0.5], [0.25, 0.0]], dtype=F64))
    torch.testing.assert_close(g, P.sigmoid(torch.tensor([[2.0, 0.5, 0.25, -3.0]], dtype=F64)))


def test_plain_expert_clamps_the_gate_from_above_and_the_other_from_both_sides():
    w = {"e.gate": torch.eye(3, dtype=F64), "e.up": torch.diag(torch.tensor([1.0, 1.0, -1.0], dtype=F64)), "e.down": torch.eye(3, dtype=F64)}
    h = torch.tensor([[5.0, -4.0, 3.0]], dtype=F64)
    g, u = torch.tensor([2.0, -4.0, 2.0], dtype=F64), torch.tensor([2.0, -2.0, -2.0], dtype=F64)
    torch.testing.assert_close(P.clamped_expert(h, w, "e.", 2.0)[0], g * P.sigmoid(1.702 * g) * (u + 1.0))


def test_plain_rotation_pairs_the_halves():
    x = torch.arange(1.0, 7.0, dtype=F64).view(1, 1, 6).repeat(4, 1, 1)
    rot = {"dims": 4, "base": 100.0}
    y = P.rotate_halves(x, rot)
    torch.testing.assert_close(y[0], x[0])
    torch.testing.assert_close(y[:, :, 4:], x[:, :, 4:])
    a0, a1 = 3.0, 3.0 * 0.1
    want = [1 * math.cos(a0) - 3 * math.sin(a0), 2 * math.cos(a1) - 4 * math.sin(a1), 3 * math.cos(a0) + 1 * math.sin(a0),
            4 * math.cos(a1) + 2 * math.sin(a1)]
    torch.testing.assert_close(y[3, 0, :4], torch.tensor(want, dtype=F64))
    stretched = P.rotate_halves(x, dict(rot, scaling={"factor": 4.0, "original": 1000, "fast": 1e9, "slow": 1e-9}))
    torch.testing.assert_close(stretched[0, :, :4], x[0, :, :4] * (0.1 * math.log(4.0) + 1.0))     # the turned part alone
    torch.testing.assert_close(stretched[0, :, 4:], x[0, :, 4:])
