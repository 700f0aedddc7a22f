"""Dinutar without a GPU: configuration, tensor names, lanes and state, the rotation's table, identities of the plain
mechanisms, and how much a fault of each mechanism would show in the logits of the test configurations."""
from __future__ import annotations

import copy
import math

import pytest
import torch

from tests import dinutar_cases as cases
from tests.plain import dinutar_plain as plain

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_config_round_trip_declared_tensors_and_lanes(name, tmp_path):
    from cpmcu_b200.models.model import Model
    from cpmcu_b200.registry import architecture, load_config

    cfg = cases.CONFIGS[name]()
    folder = cases.write_folder(cfg, cases.random_weights(cfg, 1), str(tmp_path / name))
    arch, typed = load_config(folder)
    assert arch is architecture("Dinutar")
    assert arch.config_class.from_dict(typed.to_dict()) == typed
    model = Model(arch.model_spec(typed), None)
    specs, shapes = model.weight_specs(), cases.tensor_shapes(cfg)
    assert set(specs) == set(shapes)
    assert all(tuple(specs[k].shape) == tuple(shapes[k]) for k in shapes)
    # a layer with rows or a state of its own has a lane of its own; a reader runs on its source's lane and never writes;
    # the embedding's lane lies behind them
    lane_of = {}
    for i, (layer, run) in enumerate(zip(cfg["layers"], model.schedule)):
        src = layer["mixer"].get("kv_from")
        if src is None:
            lane_of[i] = run.lane
            assert run.writes_cache
        else:
            assert run.lane == lane_of[src] and not run.writes_cache
    assert sorted(lane_of.values()) == list(range(len(lane_of))) and model.embedding_lane == len(lane_of)
    needs = model.cache_needs()
    assert len(needs) == len(lane_of) + 1
    for i, lane in lane_of.items():
        m, n = cfg["layers"][i]["mixer"], needs[lane]
        if cfg["layers"][i]["type"] == "retention":
            assert n.kv_heads == 0 and n.state["matrix_state"][0] == (m["heads"], m["dim"], m["vdim"])
        else:
            assert (n.kv_heads, n.head_dim, n.values, n.window) == (1, m["kv_rank"] + m["rot_dim"], False, None)
    state = needs[-1].state
    assert (state == {"previous_token": ((), torch.int32)}) if cfg["embedding"].get("bigram") else (state == {})
    assert model.recordable_prompt()


def test_workspace_is_measured_without_notes():
    from cpmcu_b200.ops.dry import measure_weights, measure_workspace
    from cpmcu_b200.registry import architecture

    arch = architecture("Dinutar")
    for name in sorted(cases.CONFIGS):
        spec = arch.model_spec(arch.config_class.from_dict(cases.CONFIGS[name]()))
        for dtype in (torch.float32, torch.bfloat16):
            persistent, frame, notes = measure_workspace(spec, dtype, 256, 8, 1024)
            assert persistent > 0 and frame > 0 and not notes, notes
            assert measure_weights(spec, dtype) > 0


def test_config_errors_are_collected():
    from cpmcu_b200.config.base import ConfigError
    from cpmcu_b200.config.dinutar import DinutarConfig

    bad = copy.deepcopy(cases.config_a())
    bad["layers"][1]["mixer"]["decay"] = [0.5]
    bad["layers"][1]["mixer"]["rot"]["dims"] = 26                # beyond the head
    bad["layers"][4]["mixer"]["rot"]["dims"] = 6                 # the rotated part of a latent layer is all of rot_dim
    bad["layers"][0]["mlp"]["kind"] = "gated"
    bad["embedding"]["bigram"]["buckets"] = 0
    del bad["norm"]
    with pytest.raises(ConfigError) as e:
        DinutarConfig.from_dict(bad)
    text = str(e.value)
    assert all(word in text for word in ("decay", "rot.dims", "rot_dim", "kind", "buckets", "norm"))
    for src in (1, 2, 5, 6, 9):                                  # a retention layer, a reader, the layer itself, a later one, none
        bad = copy.deepcopy(cases.config_a())
        bad["layers"][5]["mixer"]["kv_from"] = src
        with pytest.raises(ConfigError) as e:
            DinutarConfig.from_dict(bad)
        assert "kv_from" in str(e.value)
    for key, value in (("kv_rank", 25), ("rot_dim", 6)):
        bad = copy.deepcopy(cases.config_a())
        bad["layers"][5]["mixer"][key] = value
        if key == "rot_dim":
            bad["layers"][5]["mixer"]["rot"] = dict(bad["layers"][5]["mixer"]["rot"], dims=value)
        with pytest.raises(ConfigError) as e:
            DinutarConfig.from_dict(bad)
        assert "differs" in str(e.value)


ROTATIONS = [(32, 20000.0, (4.0, 512, 32.0, 1.0)), (6, 50.0, (1.5, 10, 3.0, 2.0)), (16, 5000.0, (16.0, 64, 8.0, 0.5)), (8, 100.0, None),
             (64, 1e6, (2.0, 4096, 100.0, 50.0)), (2, 10.0, (3.0, 100, 1.0, 1.0))]


@pytest.mark.parametrize("dims,base,scaling", ROTATIONS)
def test_rotation_table_against_the_plain_frequencies(dims, base, scaling):
    from cpmcu_b200.parts.position import YarnRotary

    rot = {"dims": dims, "base": base}
    params = {}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
        params = rot["scaling"]
    table, magnitude, rot_dim = YarnRotary(None, dims + 4, base, dims, **params).rotary()
    assert rot_dim == dims
    assert torch.allclose(table.double(), plain.frequencies(rot), rtol=1e-7, atol=0)
    assert abs(magnitude - plain.magnitude(rot)) < 1e-12


def test_plain_frequencies_stay_ramp_and_stretch():
    rot = {"dims": 32, "base": 1000.0}
    f = plain.frequencies(rot)
    g = plain.frequencies(dict(rot, scaling={"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}))
    turns = 256 * f / (2 * math.pi)                              # what each wave makes over the original length
    ratio = g / f
    assert torch.allclose(ratio[0], torch.tensor(1.0, dtype=F64)) and torch.allclose(ratio[-1], torch.tensor(0.25, dtype=F64))
    assert (ratio[1:] <= ratio[:-1] + 1e-12).all() and ((ratio > 0.26) & (ratio < 0.99)).any()
    assert (ratio[turns > 24.0] == 1.0).all() and torch.allclose(ratio[turns < 0.6], torch.tensor(0.25, dtype=F64))


def test_plain_rotation_pairs_halves_and_scales_by_the_magnitude():
    rot = {"dims": 4, "base": 100.0}
    x = torch.zeros(3, 1, 6, dtype=F64)
    x[:, 0, 0] = 1.0                 # the first member of pair 0 (0, 2)
    x[:, 0, 3] = 2.0                 # the second member of pair 1 (1, 3)
    x[:, 0, 5] = 7.0                 # beyond the rotated part
    y = plain.rotate_half(x, rot)
    f = [1.0, 100.0 ** -0.5]
    for p in range(3):
        want = [math.cos(p * f[0]), -2 * math.sin(p * f[1]), math.sin(p * f[0]), 2 * math.cos(p * f[1]), 0.0, 7.0]
        assert torch.allclose(y[p, 0], torch.tensor(want, dtype=F64))
    sc = {"factor": 8.0, "original": 1e6, "fast": 1e-3, "slow": 1e-4}      # every frequency is fast: only the magnitude acts
    z = plain.rotate_half(x, dict(rot, scaling=sc))
    assert torch.allclose(z[..., :4], y[..., :4] * (0.1 * math.log(8.0) + 1.0)) and torch.equal(z[..., 4:], y[..., 4:])


def test_plain_bigram_rows():
    b = {"buckets": 13, "mul_prev": 5, "mul_cur": 3}
    assert plain.bigram_rows([2, 7, 0, 1], b) == [13, (2 * 5 + 7 * 3) % 13, (7 * 5) % 13, 3]
    big = {"buckets": 1_000_003, "mul_prev": 2_000_000_011, "mul_cur": 1_999_999_973}
    assert plain.bigram_rows([76, 75], big)[1] == (76 * 2_000_000_011 + 75 * 1_999_999_973) % 1_000_003


def test_plain_retention_in_pieces_and_against_its_sum():
    g = torch.Generator().manual_seed(3)
    T, H, d, dv = 11, 2, 5, 3
    q, k = torch.randn(T, H, d, generator=g, dtype=F64), torch.randn(T, H, d, generator=g, dtype=F64)
    v = torch.randn(T, H, dv, generator=g, dtype=F64)
    decay = torch.tensor([0.5, 0.99], dtype=F64)
    whole, S = plain.retention_recurrence(q, k, v, decay)
    first, S1 = plain.retention_recurrence(q[:4], k[:4], v[:4], decay)
    rest, S2 = plain.retention_recurrence(q[4:], k[4:], v[4:], decay, state=S1)
    assert torch.allclose(torch.cat([first, rest]), whole) and torch.allclose(S2, S)
    t = 9                            # o_t = sum over s <= t of decay^(t-s) (q_t . k_s) v_s
    for h in range(H):
        want = sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
        assert torch.allclose(whole[t, h], want)


def test_plain_softmax_is_causal_and_the_join_norms_the_sum():
    p = plain.causal_softmax(torch.tensor([[0.0, 50.0], [0.0, math.log(3.0)]], dtype=F64))
    assert torch.allclose(p, torch.tensor([[1.0, 0.0], [0.25, 0.75]], dtype=F64))
    w = {"l0.ls1": torch.tensor([2.0, -1.0], dtype=F64), "l0.norm1": torch.tensor([1.0, 10.0], dtype=F64)}
    x, y = torch.tensor([[1.0, 1.0]], dtype=F64), torch.tensor([[1.0, 2.0]], dtype=F64)
    got = plain.joined(x, y, w, "l0.", 1, 3.0, 0.5)              # 3 * (1, 1) + (2, -2) = (5, 1)
    r = math.sqrt((25 + 1) / 2 + 0.5)
    assert torch.allclose(got, torch.tensor([[5 / r, 10 / r]], dtype=F64))


def _no_magnitude(monkeypatch):
    monkeypatch.setattr(plain, "magnitude", lambda rot: 1.0)


def _no_stretching(monkeypatch):
    real = plain.frequencies
    monkeypatch.setattr(plain, "frequencies", lambda rot: real({k: v for k, v in rot.items() if k != "scaling"}))


def _previous_token_lost(monkeypatch):
    monkeypatch.setattr(plain, "bigram_rows", lambda tokens, b: [b["buckets"]] * len(tokens))


def _no_layer_scale(monkeypatch):
    monkeypatch.setattr(plain, "joined", lambda x, y, w, p, which, alpha, eps: plain.rms_norm(alpha * x + y, w[f"{p}norm{which}"], eps))


def _state_lost_at_a_tile(monkeypatch):
    real = plain.retention_recurrence

    def cut(q, k, v, decay, state=None):
        return torch.cat([real(q[:64], k[:64], v[:64], decay)[0], real(q[64:], k[64:], v[64:], decay)[0]]), None
    monkeypatch.setattr(plain, "retention_recurrence", cut)


def _one_key_late(monkeypatch):
    def soft(s):
        T = s.shape[0]
        hide = torch.ones(T, T, dtype=torch.bool).triu(0)
        hide[0, 0] = False
        s = s.masked_fill(hide, float("-inf"))
        return torch.softmax(s, -1)
    monkeypatch.setattr(plain, "causal_softmax", soft)


def _a_reader_one_row_off(monkeypatch):
    real = plain.latent_attention

    def wrong(h, w, p, m, rows):
        if m.get("kv_from") is not None:
            rows = (rows[0].roll(1, 0), rows[1].roll(1, 0))
        return real(h, w, p, m, rows)
    monkeypatch.setattr(plain, "latent_attention", wrong)


@pytest.mark.parametrize("fault,names", [
    (_no_magnitude, ["a", "d", "latent_attention"]), (_no_stretching, ["a", "latent_attention"]),
    (_previous_token_lost, ["a", "c", "d"]), (_no_layer_scale, ["a", "b", "c", "d"]), (_state_lost_at_a_tile, ["a", "b", "d", "retention"]),
    (_one_key_late, ["a", "latent_attention"]), (_a_reader_one_row_off, ["a", "latent_attention"])])
def test_a_fault_of_a_mechanism_would_show(fault, names, monkeypatch):
    """The tolerances the engine is held to lie below what a fault of the mechanism would do to the logits: in 32-bit for
    most rows, in bfloat16 for the worst row (a mistake planted in the plain implementation)."""
    for name in names:
        cfg = cases.CONFIGS[name]()
        w = cases.random_weights(cfg, 11)
        ids = cases.random_ids(cfg["vocab"], 90, 5)
        want = plain.forward(cfg, w, ids)
        with monkeypatch.context() as mp:
            fault(mp)
            got = plain.forward(cfg, w, ids)
        e = cases.row_errors(got, want)[70:]
        assert float(e.median()) > 10 * cases.MEDIAN_TOL["float32"], (name, float(e.median()))
        assert float(e.max()) > cases.MEDIAN_TOL["bfloat16"], (name, float(e.max()))
