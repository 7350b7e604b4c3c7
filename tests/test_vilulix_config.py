"""Vilulix's configuration, run order, tensor names and cache needs, the cut of a step into chunks, and
its plain implementation's mechanisms against hand-made cases. No GPU."""

import json
import math

import pytest
import torch

import plain_vilulix as plain
from atomserve_b200.config.model_config import ModelConfigError
from atomserve_b200.config.registry import config_from_dict
from atomserve_b200.ops.delta import cut_into_chunks
from atomserve_b200.parts.model import build_model
from tiny_vilulix import VILULIX

F64 = torch.float64


@pytest.mark.parametrize("name", list(VILULIX))
def test_configuration_round_trips_and_names_the_plain_tensors(name):
    cfg, _ = VILULIX[name]
    arch, config = config_from_dict(json.loads(json.dumps(cfg)))
    assert arch.name == "Vilulix" and config.to_dict() == cfg
    model = build_model(arch.build_spec(config))
    have = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    assert have == plain.tensor_shapes(cfg)


def test_run_order_and_what_each_entry_keeps():
    cfg, _ = VILULIX["a"]
    arch, config = config_from_dict(cfg)
    assert config.run_order() == [(0, None), (1, None), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert [(i, opens is not None) for i, opens in config.run_order()] == plain.run_order(cfg)
    spec = arch.build_spec(config)
    assert [c.layer for c in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [c.before for c in spec.schedule] == [None, None, None, (0, 1), None, (0, 2), None, None]
    needs = build_model(spec).cache_requirements()
    assert len(needs) == 8  # every run of a layer keeps pages or state of its own
    assert [pages is not None for pages, _ in needs] == [True, True, False, True, False, True, False, True]
    assert [[s.name for s in states] for _, states in needs][:3] == [["s", "conv"], [], ["s", "n", "top"]]
    # keys of 24 and values of 16 run at 24, keys of 16 and values of 32 at 32; a latent's page holds its turned part too
    assert needs[0][0].tensors[0].width == 24 and needs[0][0].window == 20 and needs[7][0].tensors[1].width == 32
    assert needs[1][0].tensors[0].width == 48 and needs[1][0].window is None
    conv = needs[0][1][1]
    assert conv.shape == (3, 2 * 2 * 16 + 4 * 40) and needs[0][1][0].shape == (4, 16, 40)
    no_loop, _ = VILULIX["b"]
    arch, config = config_from_dict(no_loop)
    spec = arch.build_spec(config)
    assert spec.stream_steps == () and all(c.before is None for c in spec.schedule)
    assert "l2.norm2" in spec.ignored_tensors
    once = dict(VILULIX["d"][0], loop=dict(start=0, stop=2, times=1))
    arch, config = config_from_dict(once)
    assert arch.build_spec(config).stream_steps == ()  # a single pass opens with nothing


@pytest.mark.parametrize("change,words", [
    (lambda c: c["layers"][0].__setitem__("type", "attention"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 4), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("kv_heads", 3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("conv", 0), "tap"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 7), "even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].__setitem__("size", 0), "positive"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 10), "even and at most 8"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("gate_cap", 0.0), "gate_cap"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "dense"),
    (lambda c: c["loop"].__setitem__("stop", 9), "does not fit"),
    (lambda c: c["loop"].__setitem__("times", 0), "does not fit"),
    (lambda c: c.__setitem__("logit_softcap", -1.0), "positive"),
    (lambda c: c.pop("norm"), "norm"),
])  # fmt: skip
def test_rejections(change, words):
    cfg = json.loads(json.dumps(VILULIX["a"][0]))
    change(cfg)
    with pytest.raises(ModelConfigError, match=words):
        config_from_dict(cfg)


def test_cut_of_a_step_into_chunks():
    """Requests above the limit only, chunks of their own rows in order, passes of a bounded size over
    which a request may stretch."""
    assert cut_into_chunks([1, 30, 24, 70, 1], 32, 24, 100) == [([1, 55, 87, 119], [30, 32, 32, 6], [[1, 0, 1], [3, 1, 3]])]
    assert cut_into_chunks([5, 24, 1], 64, 24, 100) == []
    cut = cut_into_chunks([200, 65], 64, 24, 3)
    assert cut == [([0, 64, 128], [64, 64, 64], [[0, 0, 3]]), ([192, 200, 264], [8, 64, 1], [[0, 0, 1], [1, 1, 2]])]
    for lens in ([25, 64, 65, 128, 3, 600], [1000]):
        passes = cut_into_chunks(lens, 64, 24, 4)
        rows = [r for p in passes for start, n in zip(p[0], p[1]) for r in range(start, start + n)]
        starts = [sum(lens[:i]) for i in range(len(lens))]
        assert rows == [r for s, n in zip(starts, lens) if n > 24 for r in range(s, s + n)]
        assert all(sum(c for _, _, c in p[2]) == len(p[0]) <= 4 for p in passes)


def test_a_term_of_one_in_the_denominator():
    p = plain.softmax_and_one(torch.tensor([0.0, 0.0, math.log(2.0)], dtype=F64))
    assert torch.allclose(p, torch.tensor([0.2, 0.2, 0.4], dtype=F64))
    p = plain.softmax_and_one(torch.tensor([-800.0, -900.0], dtype=F64))  # scores far below the sink's: hardly any weight
    assert float(p.sum()) < 1e-300
    p = plain.softmax_and_one(torch.tensor([800.0, 0.0], dtype=F64))
    assert torch.allclose(p, torch.tensor([1.0, 0.0], dtype=F64))


def test_window_edges_by_hand():
    """Values that count positions, equal scores of 0: position i averages the last `window` ones, with
    one more term in the denominator."""
    n = 6
    q, k = torch.zeros(n, 1, 2, dtype=F64), torch.zeros(n, 1, 2, dtype=F64)
    v = torch.arange(n, dtype=F64)[:, None, None]
    out = plain.attend_window(q, k, v, 1.0, 3)[:, 0, 0]
    assert torch.allclose(out, torch.tensor([0.0, 1 / 3, 3 / 4, 6 / 4, 9 / 4, 12 / 4], dtype=F64))
    assert torch.allclose(plain.attend_window(q, k, v, 1.0, None)[5, 0, 0], torch.tensor(15 / 7, dtype=F64))


def test_a_written_value_is_replaced_and_read_at_once():
    """Keys e_0, e_0, e_1 with beta 1 and no decay: the second write replaces the first, the third leaves
    it alone, and every token reads what it has just written; then a decay halves what is held before
    the token's correction."""
    q = k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]], [[0.0, 1.0]]], dtype=F64)
    v = torch.tensor([[[3.0]], [[5.0]], [[7.0]]], dtype=F64)
    one = torch.ones(3, 1, dtype=F64)
    o, S = plain.delta_recurrence(q, k, v, one, one)
    assert o.flatten().tolist() == [3.0, 5.0, 7.0] and S.flatten().tolist() == [5.0, 7.0]
    o, S = plain.delta_recurrence(q, k, v, 0.5 * one, 0.5 * one)
    assert o.flatten().tolist() == [1.5, 0.75 + 0.5 * (5.0 - 0.75), 3.5]
    assert torch.allclose(S.flatten(), torch.tensor([0.5 * (0.75 + 0.5 * 4.25), 3.5], dtype=F64))


def test_convolution_by_hand():
    x, taps = torch.tensor([[1.0], [2.0], [4.0]], dtype=F64), torch.tensor([[10.0, 1.0]], dtype=F64)
    assert plain.causal_convolution(x, taps).flatten().tolist() == [1.0, 12.0, 24.0]  # the last tap is the current token's


def test_gains_are_stored_around_zero_and_passes_add_the_embedding():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    assert torch.allclose(plain.centred_gain_norm(x, torch.tensor([0.0, 1.0]), 0.0), torch.tensor([[3.0, 8.0]], dtype=F64) / 12.5**0.5)
    cfg, _ = VILULIX["d"]
    w = plain.random_checkpoint(cfg, 1)
    for name in w:  # without sublayers' outputs only the embedding is left, added once more by the second pass
        if name.endswith((".o", ".down")):
            w[name] = torch.zeros_like(w[name])
    layers = []
    plain.forward([5, 9], w, cfg, streams=layers)
    x0 = w["embed"][[5, 9]].double()
    assert all(torch.equal(s, f * x0) for s, f in zip(layers, (1, 1, 2, 2)))
