"""Lomopel without a GPU: the parser and what it refuses, the tensor plan with its free sizes, and the plain implementation
against itself - that leaving out any one mechanism moves its logits far beyond rounding, so that the GPU tests' bounds mean
something."""
import copy

import pytest
import torch

import tiny_lomopel as tl
from helpers import load_plain, random_tokens
from plain_lomopel import (PlainLomopel, convolved, delta_step, gelu_tanh, in_window, mixed_value, rotate, softmax_read,
                           temperature, whole_sequence)

from nanoinfer_b200.config import config_from_dict
from nanoinfer_b200.config.model_config import ConfigError
from nanoinfer_b200.parts.base import FreeDim
from nanoinfer_b200.weights.loader import WeightError, check_tensors
from nanoinfer_b200.weights.plan import tensor_plan

F64 = torch.float64


def test_parser_reads_every_size_and_constant():
    cfg = config_from_dict(tl.L1)
    assert cfg.architecture == "Lomopel" and cfg.hidden_size == 96 and cfg.vocab_size == 300
    assert cfg.embedding.kind == "table" and cfg.embedding.extra_dict() == {"row_scale": 6.0}
    p, a, b, c = cfg.layers[0], cfg.layers[1], cfg.layers[2], cfg.layers[4]
    assert p.arrangement == "pre_norm" and p.extra_dict()["layer_scale"] and p.mixer_norm.kind == "rmsnorm_one_plus"
    assert p.mixer_norm.eps == 1e-5
    sides = p.mixer.extra_dict()
    assert p.mixer.kind == "parallel_mixers" and (sides["left_scale"], sides["right_scale"], sides["join"]) == (1.3, 0.7, True)
    left, right = sides["left"], sides["right"]
    assert (left.kind, left.window, left.position.kind, left.position.rotary_dim, left.position.theta) == \
        ("normed_qk_attention", 20, "rope_exact", 12, 50000.0)
    assert left.position.pairing == "half" and left.extra_dict()["element_gate"] and left.extra_dict()["head_unit_norm"]
    assert not left.extra_dict()["bias"]
    e = right.extra_dict()
    assert (right.kind, right.num_heads, right.num_kv_heads, right.head_dim, e["value_dim"], e["conv_taps"]) == ("gated_delta", 6, 2, 20, 12, 4)
    assert (e["decay"], e["gate"]) == ("key_channel", "low_rank_sigmoid")
    e = a.mixer.extra_dict()
    assert (a.mixer.num_heads, a.mixer.num_kv_heads, a.mixer.head_dim, e["value_dim"], a.mixer.softmax_scale) == (4, 2, 24, 40, 0.15)
    assert e["sink"] == "learned" and e["temperature"] == (0.3, 16.0) and e["bias"] and e["output_bias"] and a.mixer.window is None
    assert [layer.mixer.extra_dict().get("value_mix") for layer in cfg.layers] == [None, "first", None, None, "later", "later"]
    assert c.mixer.extra_dict()["temperature"] is None and b.feed_forward is None and b.ffn_norm is None
    assert a.feed_forward.kind == "swiglu" and a.feed_forward.extra_dict()["activation"] == "gelu_tanh"


def test_tensor_plan_has_the_layers_own_tensors():
    plan = {p.name: p for p in tensor_plan(config_from_dict(tl.L1))}
    assert plan["l1.mix.q.b"].shape == (96,) and plan["l1.mix.o.b"].shape == (96,) and plan["l1.mix.sink"].shape == (4,)
    assert plan["l1.mix.vmix"].shape == () and "l2.mix.vmix" not in plan and "l0.mix.left.sink" not in plan
    assert plan["l0.mix.left.g"].shape == (6 * 24, 96) and plan["l0.mix.right.dt_bias"].shape == (6 * 20,)
    assert plan["l0.mix.right.A_log"].shape == (6,) and plan["l0.mix.right.q"].shape == (2 * 20, 96)
    assert plan["l0.ls1"].shape == (96,) and "l0.ls2" in plan and "l2.ls1" in plan and "l2.ls2" not in plan and "l2.norm2" not in plan
    a1 = plan["l0.mix.right.a1"].shape
    assert isinstance(a1[0], FreeDim) and a1[1] == 96 and isinstance(plan["l0.mix.right.g2"].shape[1], FreeDim)


def test_thin_matrices_take_their_size_from_the_tensors():
    cfg = config_from_dict(tl.L1)
    found = {p.name: tuple(int(n) for n in p.shape) for p in tensor_plan(cfg)}
    check_tensors("m", cfg, found)                                     # the sizes random weights are made with
    found["l0.mix.right.a1"], found["l0.mix.right.a2"] = (13, 96), (120, 13)
    found["l0.mix.right.g1"], found["l0.mix.right.g2"] = (1, 96), (72, 1)
    check_tensors("m", cfg, found)                                     # another size each, and another layer keeps its own
    for bad in ({"l0.mix.right.a2": (120, 12)}, {"l0.mix.right.a1": (13, 95)}, {"l0.mix.right.g1": (0, 96), "l0.mix.right.g2": (72, 0)}):
        with pytest.raises(WeightError):
            check_tensors("m", cfg, {**found, **bad})
    extra = {**found, "l2.norm2": (96,), "l2.ls2": (96,), "l2.mix.vmix": ()}
    check_tensors("m", cfg, extra)                                     # stored beside a layer that has no use for them
    with pytest.raises(WeightError):
        check_tensors("m", cfg, {**found, "l2.other": (1,)})


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "not a mixer"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=11), "even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "positive"),
    (lambda c: c["layers"][5]["mixer"].update(vdim=39), "one size"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(conv=0), "positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not supported"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_parser_refuses(change, message):
    raw = copy.deepcopy(tl.L1)
    change(raw)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(raw)


def test_small_functions():
    assert in_window(30, 11, 20) and not in_window(30, 10, 20) and in_window(5, 5, 1) and not in_window(5, 4, 1) and not in_window(4, 5, 9)
    t = {"coef": 0.5, "every": 4}
    assert temperature(t, 2) == 1.0 and abs(temperature(t, 3) - (1 + 0.5 * 0.6931471805599453)) < 1e-12 and temperature(None, 99) == 1.0
    assert temperature(t, 6) == temperature(t, 3) < temperature(t, 7)
    zero = torch.tensor(0.0, dtype=F64)
    v = [torch.tensor([2.0], dtype=F64)]
    assert softmax_read([zero], v).item() == 2.0 and abs(softmax_read([zero], v, 0.0).item() - 1.0) < 1e-12
    assert softmax_read([zero], v, -80.0).item() > 1.999999 and softmax_read([zero], v, 800.0).item() == 0.0
    x = torch.tensor([1.0, 2.0, 3.0], dtype=F64)
    assert mixed_value(x, 3 * x, 0.25).tolist() == [1.5, 3.0, 4.5]
    r = rotate(torch.tensor([1.0, 0.0, 0.0, 1.0, 7.0], dtype=F64), 1, {"dims": 4, "base": 1.0})
    c, s = torch.cos(torch.tensor(1.0, dtype=F64)), torch.sin(torch.tensor(1.0, dtype=F64))
    torch.testing.assert_close(r, torch.stack([c, -s, s, c, torch.tensor(7.0, dtype=F64)]))
    torch.testing.assert_close(gelu_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"))
    past = [torch.zeros(1, dtype=F64), torch.ones(1, dtype=F64)]
    y = convolved(torch.full((1,), 2.0, dtype=F64), torch.tensor([[1.0, 10.0, 100.0]], dtype=F64), past)
    assert abs(y.item() - 210.0) < 1e-9 and [p.item() for p in past] == [1.0, 2.0]
    S = torch.tensor([[1.0], [2.0]], dtype=F64)
    k, q, v1 = torch.tensor([1.0, 0.0], dtype=F64), torch.tensor([0.0, 1.0], dtype=F64), torch.tensor([5.0], dtype=F64)
    S2, o = delta_step(S, torch.tensor([0.5, 0.25], dtype=F64), 1.0, q, k, v1)
    assert S2.view(-1).tolist() == [5.0, 0.5] and o.item() == 0.5       # row by row decay; the error is written under k


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    d = str(tmp_path_factory.mktemp("lomopel") / "l1")
    tl.write_model(d, tl.L1, 11, ranks=tl.RANKS["L1"])
    return load_plain(d)


def test_token_by_token_state_carries_everything(model):
    """Two halves fed one after the other through one state give what the whole sequence gives."""
    cfg, w = model
    toks = random_tokens(cfg["vocab"], 60, 3)
    want = whole_sequence(cfg, w, toks)
    plain = PlainLomopel(cfg, w)
    st = plain.new_state()
    assert torch.equal(torch.cat([plain.run(toks[:29], st), plain.run(toks[29:], st)]), want)


@pytest.mark.parametrize("what", ["sink", "q_temp", "v_mix", "embedding_scale", "ls1", "ls2", "window", "rotation", "gate", "scales",
                                  "biases", "output_bias", "conv", "decay", "channel", "beta", "thin_gate", "read_norm", "one_plus",
                                  "first_mixing"])
def test_every_mechanism_moves_the_logits(model, what):
    """Without it (or with a slightly wrong one) the plain logits at the end of a 50-token prompt (8 tokens for the sink) move
    by far more than any rounding."""
    cfg, w = model
    toks = random_tokens(cfg["vocab"], 8 if what == "sink" else 50, 5)
    want = whole_sequence(cfg, w, toks)[-1]
    cfg2, w2, leave = copy.deepcopy(cfg), dict(w), None
    lefts = [cfg2["layers"][i]["mixer"]["left"] for i in (0, 3)]

    def each(suffix, f):
        for name in list(w):
            if name.endswith(suffix):
                w2[name] = f(w[name])

    if what in ("sink", "q_temp", "v_mix", "embedding_scale", "ls1", "ls2"):
        leave = what
    elif what == "window":
        for m in lefts:
            m["mask"]["size"] += 1
    elif what == "rotation":
        for m in lefts:
            m["rot"]["base"] = 30.0
    elif what == "gate":
        each("left.g", torch.zeros_like)
    elif what == "scales":
        cfg2["layers"][0]["mixer"]["left_scale"] = cfg2["layers"][3]["mixer"]["right_scale"] = 1.0
    elif what == "biases":
        for s in (".q.b", ".k.b", ".v.b"):
            each(s, torch.zeros_like)
    elif what == "output_bias":
        each(".o.b", torch.zeros_like)
    elif what == "conv":
        each(".conv", lambda t: t.flip(1))
    elif what == "decay":
        each(".A_log", lambda t: t + 1.0)
    elif what == "channel":
        each(".dt_bias", lambda t: t.roll(1))                           # another channel's decay
    elif what == "beta":
        each("right.b", torch.zeros_like)
    elif what == "thin_gate":
        each(".g2", torch.zeros_like)
    elif what == "read_norm":
        each("right.norm", torch.ones_like)
    elif what == "one_plus":
        each(".norm2", lambda t: t - 1.0)
    elif what == "first_mixing":
        cfg2["layers"][2]["mixer"].update(v_mix=False)
        cfg2["layers"][1]["mixer"]["v_mix"] = False                     # another layer becomes the first one
    plain = PlainLomopel(cfg2, w2)
    st = plain.new_state()
    got = torch.stack([plain.token(int(t), st, leave_out=leave) for t in toks])[-1]
    moved = (got - want).abs().max().item()
    assert moved > 0.02 * want.abs().max().item(), f"{what}: the logits moved by {moved:.3g} only"
