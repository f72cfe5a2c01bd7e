"""Kepusun without a GPU: the parser and what it refuses, whose cache a layer reads, the tensor plan, and the plain
implementation against itself - that leaving out any one mechanism moves its logits far beyond rounding, so that the GPU
tests' bounds mean something."""
import copy
import math

import pytest
import torch

import plain_kepusun as pk
import tiny_kepusun as tk
from helpers import load_plain, random_tokens
from plain_kepusun import PlainKepusun, choose_experts, memory_step, whole_sequence

from nanoinfer_b200.config import config_from_dict
from nanoinfer_b200.config.model_config import ConfigError
from nanoinfer_b200.weights.plan import tensor_plan

F64 = torch.float64


def test_parser_reads_every_size_and_constant():
    cfg = config_from_dict(tk.U1)
    assert (cfg.architecture, cfg.hidden_size, cfg.vocab_size, cfg.streams) == ("Kepusun", 96, 300, 3)
    m, a, b, _ = cfg.layers
    assert m.arrangement == "hyper_connections" and m.extra_dict()["streams"] == 3 and m.mixer_norm.kind == "dynamic_tanh"
    assert (m.mixer.kind, m.mixer.num_heads, m.mixer.head_dim) == ("matrix_memory", 3, 20)
    assert m.mixer.extra_dict() == {"value_dim": 12, "gate_cap": 11.0, "norm_eps": 1e-5}
    e = m.feed_forward.extra_dict()
    assert (m.feed_forward.kind, m.feed_forward.intermediate_size, e["experts"], e["top"]) == ("routed_experts", 40, 6, 2)
    assert (e["unit"], e["renormalize"], e["weight_scale"], e["groups"], e["keep_groups"]) == ("relu2", True, 1.7, 3, 2)
    assert (a.mixer.kind, a.mixer.num_heads, a.mixer.num_kv_heads, a.mixer.head_dim, a.mixer.softmax_scale) == \
        ("differential_attention", 4, 2, 24, 0.3)
    assert a.mixer.extra_dict() == {"value_dim": 40, "norm_eps": 1e-5, "diff": 0.35, "own_kv": True}
    assert a.feed_forward.extra_dict()["groups"] == 1
    assert b.feed_forward is None and b.ffn_norm is None and not b.mixer.extra_dict()["own_kv"]
    assert [r.cache_of for r in cfg.schedule] == [None, None, 1, None]
    assert [r.cache_of for r in config_from_dict(tk.U4).schedule] == [None, None, 0, None, 0, None]
    third = config_from_dict(tk.U3).layers
    assert third[2].mixer.extra_dict()["value_dim"] == 8 and third[3].mixer.num_kv_heads == 3


def test_tensor_plan():
    plan = {p.name: p.shape for p in tensor_plan(config_from_dict(tk.U1))}
    assert plan["embed"] == plan["head"] == (300, 96) and plan["final.norm"] == plan["final.norm.b"] == (96,)
    assert plan["final.norm.alpha"] == plan["l0.norm1.alpha"] == ()
    assert plan["l0.mix.q"] == (60, 96) and plan["l0.mix.v"] == plan["l0.mix.g"] == (36, 96) and plan["l0.mix.norm"] == (36,)
    assert plan["l0.mix.i"] == (3, 96) and plan["l0.mix.f.b"] == (3,) and plan["l0.mix.o"] == (96, 36)
    assert plan["l1.mix.q"] == (192, 96) and plan["l1.mix.k"] == (96, 96) and plan["l1.mix.v"] == (80, 96) and plan["l1.mix.lk2"] == (24,)
    assert plan["l2.mix.q"] == (288, 96) and plan["l2.mix.o"] == (96, 240) and "l2.mix.k" not in plan and "l2.mix.v" not in plan
    assert plan["l0.hc1.mix"] == (3, 3) and plan["l0.hc2.in"] == (3,) and "l2.hc1.out" in plan
    assert not any(n in plan for n in ("l2.hc2.in", "l2.norm2", "l2.norm2.alpha", "l2.mlp.router"))
    assert plan["l0.mlp.e5.up"] == (40, 96) and plan["l0.mlp.e5.down"] == (96, 40) and "l0.mlp.e0.gate" not in plan


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "not a mixer"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "no keys and values"),
    (lambda c: c["layers"][2]["mixer"].update(dim=20), "other sizes"),
    (lambda c: c["layers"][0]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "not supported"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_parser_refuses(change, message):
    raw = copy.deepcopy(tk.U1)
    change(raw)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(raw)


def test_small_functions():
    z = torch.tensor([3.0, 0.0, 2.9, 2.8, 1.0, 2.7], dtype=F64)
    s = torch.softmax(z, 0)
    ids, w = choose_experts(z, {"experts": 6, "top": 2, "scale": 1.0})
    assert ids == [0, 2] and abs(sum(w).item() - 1.0) < 1e-12
    ids, w = choose_experts(z, {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}})
    assert ids == [0, 1] and abs(w[0].item() - 3.0 * (s[0] / (s[0] + s[1])).item()) < 1e-12      # only the first pair may be chosen
    ids, _ = choose_experts(z, {"experts": 6, "top": 3, "scale": 1.0, "groups": {"count": 2, "keep": 1}})
    assert sorted(ids) == [0, 1, 2]
    # the stabilised memory is the plain recurrence: exp(m) S and exp(m) n follow sums of weighted products
    g = torch.Generator().manual_seed(0)
    mem = [torch.zeros(4, 3, dtype=F64), torch.zeros(4, dtype=F64), torch.zeros((), dtype=F64)]
    S, n = torch.zeros(4, 3, dtype=F64), torch.zeros(4, dtype=F64)
    for _ in range(20):
        q, k, v = (torch.randn(x, generator=g, dtype=F64) for x in (4, 4, 3))
        i, f = torch.randn(2, generator=g, dtype=F64)
        f = torch.nn.functional.logsigmoid(f)
        o = memory_step(mem, q, k, v, i, f)
        S, n = torch.exp(f) * S + torch.exp(i) * torch.outer(k, v), torch.exp(f) * n + torch.exp(i) * k
        torch.testing.assert_close(mem[0] * torch.exp(mem[2]), S)
        want = S.T @ q / (max(abs((n @ q).item()), 1.0) + 1e-6 * math.exp(mem[2].item()))
        torch.testing.assert_close(o, want)


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    d = str(tmp_path_factory.mktemp("kepusun") / "u1")
    tk.write_model(d, tk.U1, 11)
    return load_plain(d)


def test_token_by_token_state_carries_everything(model):
    """Two halves fed one after the other through one state give what the whole sequence gives."""
    cfg, w = model
    toks = random_tokens(cfg["vocab"], 50, 3)
    want = whole_sequence(cfg, w, toks)
    plain = PlainKepusun(cfg, w)
    st = plain.new_state()
    assert torch.equal(torch.cat([plain.run(toks[:23], st), plain.run(toks[23:], st)]), want)


def _zero(w, *names):
    return {**w, **{n: torch.zeros_like(w[n]) for n in names}}


@pytest.mark.parametrize("what", ["alpha", "norm bias", "norm weight", "in", "out", "mix", "mix order", "input gate", "forget gate", "cap",
                                  "normaliser", "maximum", "head norm", "norm weight of the heads", "output gate", "second map",
                                  "lambda", "diff factor", "shared keys", "groups", "over their sum", "router scale", "square",
                                  "old tokens"])
def test_every_mechanism_moves_the_logits(model, what, monkeypatch):
    """Without it the plain logits of the last tokens of a 50-token prompt move by far more than any rounding."""
    cfg, w = model
    toks = random_tokens(cfg["vocab"], 50, 5)
    want = whole_sequence(cfg, w, toks)[-12:]
    cfg2, w2 = copy.deepcopy(cfg), dict(w)
    layers = cfg2["layers"]
    if what == "alpha":
        w2["l1.norm2.alpha"] = torch.ones_like(w["l1.norm2.alpha"])
    elif what == "norm bias":
        w2 = _zero(w, "l0.norm1.b")
    elif what == "norm weight":
        w2["final.norm"] = torch.ones_like(w["final.norm"])
    elif what in ("in", "out"):
        for n in (f"l0.hc2.{what}", f"l1.hc1.{what}", f"l1.hc2.{what}", f"l2.hc1.{what}"):
            w2[n] = w[n].flip(0)                                       # the coefficients in another order
    elif what == "mix":
        w2["l1.hc2.mix"] = torch.eye(3)
    elif what == "mix order":
        w2["l0.hc1.mix"], w2["l1.hc1.mix"] = w["l0.hc1.mix"].T, w["l1.hc1.mix"].T
    elif what in ("input gate", "forget gate"):
        g = what[0]
        w2 = _zero(w, f"l0.mix.{g}", f"l3.mix.{g}")
    elif what == "cap":
        layers[0]["mixer"]["gate_cap"] = layers[3]["mixer"]["gate_cap"] = 2.0
    elif what == "normaliser":
        monkeypatch.setattr(pk, "unit_rms", lambda x, eps: x)          # (the norm per head hides most of a factor) ...
        want = whole_sequence(cfg, w, toks)[-12:]
        orig = pk.memory_step

        def no_normaliser(mem, q, k, v, i, f):
            S = orig(mem, q, k, v, i, f)
            return S * (torch.maximum((mem[1] @ q).abs(), torch.exp(-mem[2])) + 1e-6)
        monkeypatch.setattr(pk, "memory_step", no_normaliser)
    elif what == "maximum":
        monkeypatch.setattr(pk, "unit_rms", lambda x, eps: x)          # ... the floor exp(-m) of the denominator
        want = whole_sequence(cfg, w, toks)[-12:]

        def no_floor(mem, q, k, v, i, f):
            S, n = torch.exp(f) * mem[0] + torch.exp(i) * torch.outer(k, v), torch.exp(f) * mem[1] + torch.exp(i) * k
            mem[:] = [S, n, mem[2]]
            return S.T @ q / ((n @ q).abs() + 1e-6)
        monkeypatch.setattr(pk, "memory_step", no_floor)
    elif what == "head norm":
        monkeypatch.setattr(pk, "unit_rms", lambda x, eps: x)
    elif what == "norm weight of the heads":
        w2["l0.mix.norm"] = torch.ones_like(w["l0.mix.norm"])
    elif what == "output gate":
        w2 = _zero(w, "l0.mix.g", "l3.mix.g")
    elif what == "second map":
        monkeypatch.setattr(pk, "difference_weight", lambda *a: 0.0)
    elif what == "lambda":
        w2 = _zero(w, "l1.mix.lq1", "l2.mix.lq1", "l1.mix.lk2", "l2.mix.lk2")
    elif what == "diff factor":
        orig_w = pk.difference_weight
        monkeypatch.setattr(pk, "difference_weight", lambda ww, pre, diff: orig_w(ww, pre, diff) - diff + cfg["layers"][int(pre[1])]["mixer"]["diff"])
        layers[1]["mixer"]["diff"] = layers[2]["mixer"]["diff"] = 0.0
    elif what == "shared keys":
        for n in ("k", "v"):
            w2[f"l2.mix.{n}"] = w[f"l1.mix.{n}"]
        del layers[2]["mixer"]["kv_from"]                              # the same matrices over its own input instead
    elif what == "groups":
        del layers[0]["mlp"]["router"]["groups"], layers[3]["mlp"]["router"]["groups"]
    elif what == "over their sum":
        orig_c = pk.choose_experts

        def plain_scores(z, r):
            ids, _ = orig_c(z, r)
            s = torch.softmax(z, 0)
            return ids, [s[e] * r["scale"] for e in ids]
        monkeypatch.setattr(pk, "choose_experts", plain_scores)
    elif what == "router scale":
        layers[0]["mlp"]["router"]["scale"] = 1.0
    elif what == "square":
        monkeypatch.setattr(pk, "expert", lambda ww, pre, h: ww[pre + "down"] @ torch.relu(ww[pre + "up"] @ h))
    elif what == "old tokens":
        toks = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    got = whole_sequence(cfg2, w2, toks)[-12:]
    moved = (got - want).abs().max().item()
    assert moved > (0.004 if what == "old tokens" else 0.01) * want.abs().max().item(), f"{what}: the logits moved by {moved:.3g} only"
