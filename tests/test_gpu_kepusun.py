"""Kepusun on the GPU against the plain implementation (tests/plain_kepusun.py): kernels and parts alone, one-layer models
whose weights or prompts make ONE token count - far back, in prompts and in decoding -, then whole models replayed under
four ways of cutting the same requests, in 32-bit and in bfloat16, long decoding through replayed graphs, greedy
generation through the engine and the trace runner from the command line.  The models are small and of other sizes than
any real one."""
import json
import os
import subprocess
import sys

import pytest
import torch

import plain_kepusun as pk
import replay_util as ru
import tiny_kepusun as tk
from helpers import load_plain, random_tokens
from plain_kepusun import PlainKepusun, choose_experts, memory_step, unit_rms, whole_sequence

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64
I32 = dict(dtype=torch.int32, device=DEV)
DTYPES = [torch.float32, torch.bfloat16]


def _tol(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1.6e-2, atol=1.6e-2)


def _rand(g, *shape, scale=1.0):
    return torch.randn(*shape, generator=g) * scale


# ---- the pass over residual streams ------------------------------------------------------------------------

@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8, 9, 32])
@pytest.mark.parametrize("d", [64, 76, 50, 516])
@pytest.mark.parametrize("dtype", DTYPES)
def test_streams_over_two_sublayers_and_the_final_sum(dtype, d, streams):
    """From the embedding's rows through a plain output and then routed rows to the sum at some rows: every stream and
    every input against the equations, written out."""
    from nanoinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(streams * 1000 + d)
    T, top = 7, 3
    base = _rand(g, T, d)
    ins = [_rand(g, streams, scale=0.5) for _ in range(2)]
    mixes = [_rand(g, streams, streams, scale=0.5) for _ in range(2)]
    outs = [_rand(g, streams) for _ in range(2)]
    norms = [(torch.tensor([0.7]), 1 + _rand(g, d, scale=0.3), _rand(g, d, scale=0.2)) for _ in range(3)]
    dev = lambda *ts: tuple(t.to(DEV) for t in ts)
    st = ops.ResidualStreams(base.to(DEV), streams)
    X = [base.double() for _ in range(streams)]

    def want(x, coef, norm):
        u = sum((coef[s].double() if coef is not None else 1.0) * v for s, v in enumerate(x))
        return u, torch.tanh(norm[0].double() * u) * norm[1].double() + norm[2].double()

    h = st.read(ins[0].to(DEV), dev(*norms[0]), dtype)
    torch.testing.assert_close(h.cpu().double(), want(X, ins[0], norms[0])[1], **_tol(dtype))
    y = _rand(g, T, d)
    st.leave(y.to(DEV), mixes[0].to(DEV), outs[0].to(DEV))
    X = [sum(mixes[0][s, t].double() * X[s] for s in range(streams)) + outs[0][t].double() * y.double() for t in range(streams)]
    u = st.read(ins[1].to(DEV))                                  # without a norm: the FP32 sum itself
    torch.testing.assert_close(u.cpu().double(), want(X, ins[1], norms[1])[0], rtol=2e-5, atol=1e-4)
    torch.testing.assert_close(st.x.cpu().double(), torch.stack(X, 1), rtol=2e-5, atol=1e-4)
    z = _rand(g, T * top, d).to(dtype)
    ids = torch.randint(0, 5, (T, top), generator=g)
    wts = torch.rand(T, top, generator=g)
    where = torch.randperm(T * top, generator=g)
    st.leave(ops.RoutedRows(z.to(DEV), ids.to(**I32), wts.to(DEV), where.to(**I32)), mixes[1].to(DEV), outs[1].to(DEV))
    y2 = (wts.double()[..., None] * z.double()[where].view(T, top, d)).sum(1)
    X = [sum(mixes[1][s, t].double() * X[s] for s in range(streams)) + outs[1][t].double() * y2 for t in range(streams)]
    rows = torch.tensor([6, 0, 3])
    before = st.x.clone()
    h = st.read(None, dev(*norms[2]), dtype, rows=rows.to(**I32))
    torch.testing.assert_close(h.cpu().double(), want(X, None, norms[2])[1][rows], **(_tol(dtype) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=1e-4)))
    assert torch.equal(before, st.x)                             # reading some rows leaves the streams as they are
    # experts' rows for every (token, expert)
    z = _rand(g, T * 5, d).to(dtype)
    st.pending = None
    st.leave(ops.RoutedRows(z.to(DEV), ids.to(**I32), wts.to(DEV), None, all_experts=5), mixes[1].to(DEV), outs[1].to(DEV))
    y3 = (wts.double()[..., None] * torch.gather(z.double().view(T, 5, d), 1, ids[..., None].expand(-1, -1, d))).sum(1)
    st.read(ins[0].to(DEV), dev(*norms[0]), dtype)
    old = before.cpu().double()
    want_x = torch.einsum("st,nsd->ntd", mixes[1].double(), old) + outs[1].double()[None, :, None] * y3[:, None]
    torch.testing.assert_close(st.x.cpu().double(), want_x, rtol=2e-5, atol=2e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_tanh_norm_as_an_ordinary_norm(dtype):
    """The norm part in a pre-norm place: the pending addition joins the stream, selected rows leave it alone."""
    from nanoinfer_b200.config.model_config import NormSpec
    from nanoinfer_b200.engine.runtime import Runtime
    from nanoinfer_b200.parts.norm import DynamicTanh
    g = torch.Generator().manual_seed(3)
    d, T = 72, 9
    w = {"weight": 1 + _rand(g, d, scale=0.3), "b": _rand(g, d, scale=0.3), "alpha": torch.tensor(0.8)}
    norm = DynamicTanh(NormSpec("dynamic_tanh", 1e-5), d, w, Runtime(device=torch.device(DEV), dtype=dtype, page_size=16))
    h, delta = _rand(g, T, d), _rand(g, T, d)
    f = lambda x: torch.tanh(0.8 * x.double()) * w["weight"].double() + w["b"].double()
    hd = h.to(DEV)
    rows = torch.tensor([8, 2], **I32)
    torch.testing.assert_close(norm.forward(hd, delta.to(DEV), rows=rows).cpu().double(), f(h + delta)[[8, 2]], **_tol(dtype))
    assert torch.equal(hd.cpu(), h)
    torch.testing.assert_close(norm.forward(hd, delta.to(DEV)).cpu().double(), f(h + delta), **_tol(dtype))
    torch.testing.assert_close(hd.cpu(), h + delta)
    torch.testing.assert_close(norm.forward(hd, None).cpu().double(), f(h + delta), **_tol(dtype))


# ---- the matrix memory -----------------------------------------------------------------------------------------

class _Memories:
    """A matrix-memory layer's kernels driven request by request, beside the plain recurrence in FP64."""

    def __init__(self, H, D, V, dtype, slots=4, cap=9.0, seed=0):
        from nanoinfer_b200.kernels import ops
        self.ops, self.H, self.D, self.V, self.dtype, self.cap = ops, H, D, V, dtype, cap
        g = self.g = torch.Generator().manual_seed(seed)
        self.state = torch.zeros(slots, ops.mlstm_state_floats(H, D, V), device=DEV)
        self.bias_i, self.bias_f = _rand(g, H), 3.0 + _rand(g, H)
        self.weight = 1 + _rand(g, H * V, scale=0.3)
        self.plain = [None] * slots

    def fresh(self, slot):
        self.state[slot].zero_()
        self.plain[slot] = pk.fresh_memory({"heads": self.H, "dim": self.D, "vdim": self.V})

    def step(self, lens, slots, gate_shift=(0.0, 0.0), gate_scale=2.0):
        """Random inputs for a step of ``lens`` tokens per request; returns (got, want) [T, H V]."""
        ops, H, D, V, g = self.ops, self.H, self.D, self.V, self.g
        n = sum(lens)
        cols = 2 * H * (D + V)
        single = max(lens) == 1
        act = torch.float32 if single else self.dtype
        proj = torch.zeros(n, cols + (-cols % 8))
        proj[:, :cols] = _rand(g, n, cols)
        proj = proj.to(act)
        z = _rand(g, n, 2 * H + 3, scale=gate_scale)
        z[:, 1:1 + H] += gate_shift[0]
        z[:, 2 + H:2 + 2 * H] += gate_shift[1]
        y = torch.empty(n, H * V, dtype=self.dtype, device=DEV)
        cu = torch.tensor([0] + list(torch.cumsum(torch.tensor(lens), 0)), **I32)
        common = (proj.to(DEV), z.to(DEV), 1, 2 + H, self.bias_i.to(DEV), self.bias_f.to(DEV), self.cap, self.state, cu,
                  torch.tensor(slots, **I32), len(lens))
        rest = (D ** -0.5, self.weight.to(DEV), 1e-5)
        if single:
            ops.mlstm_token_step(*common, *rest, y, H, D, V)
        else:
            buf = torch.full((ops.mlstm_buffer_floats(n, len(lens), H, D, V),), float("nan"), device=DEV)
            out = torch.full((n, H * V), float("nan"), device=DEV)
            ops.mlstm_chunk_step(*common, max(lens), *rest, buf, out, y, H, D, V)
        x, zz = proj.double(), z.double()
        want, at = torch.zeros(n, H * V, dtype=F64), 0
        for ln, slot in zip(lens, slots):
            for t in range(at, at + ln):
                q, k = x[t, :H * D].view(H, D) * D ** -0.5, x[t, H * D:2 * H * D].view(H, D)
                v, gate = x[t, 2 * H * D:2 * H * D + H * V].view(H, V), x[t, 2 * H * D + H * V:cols]
                i = pk.capped(zz[t, 1:1 + H] + self.bias_i.double(), self.cap)
                f = torch.nn.functional.logsigmoid(pk.capped(zz[t, 2 + H:2 + 2 * H] + self.bias_f.double(), self.cap))
                o = [unit_rms(memory_step(self.plain[slot][a], q[a], k[a], v[a], i[a], f[a]), 1e-5) for a in range(H)]
                want[t] = torch.cat(o) * self.weight.double() * torch.sigmoid(gate)
            at += ln
        return y.cpu().double(), want

    def check_states(self, tol=2e-5):
        H, D, V = self.H, self.D, self.V
        rec = -(-(D * V + D) // 4) * 4
        for slot, mem in enumerate(self.plain):
            if mem is None:
                continue
            row = self.state[slot].cpu().double()
            for a, (S, n, m) in enumerate(mem):
                scale = max(1.0, S.abs().max().item())
                torch.testing.assert_close(row[a * rec:a * rec + D * V].view(D, V) / scale, S / scale, rtol=tol, atol=tol)
                torch.testing.assert_close(row[a * rec + D * V:a * rec + D * V + D] / scale, n / scale, rtol=tol, atol=tol)
                torch.testing.assert_close(row[H * rec + a], m, rtol=1e-5, atol=1e-5)


# the read-out is divided by its own root mean square, which magnifies roundings where a head reads almost nothing
def _close(got, want, dtype, label=""):
    err = (got - want).abs()
    tol = 2e-4 if dtype == torch.float32 else 3e-2
    assert torch.isfinite(got).all(), label
    assert err.max().item() <= 4 * tol * max(1.0, want.abs().max().item()), (label, err.max().item())
    assert err.pow(2).mean().sqrt().item() <= tol * want.pow(2).mean().sqrt().item(), (label, err.pow(2).mean().sqrt().item())


MEMORY_SIZES = [(3, 20, 12), (1, 16, 16), (2, 64, 128), (2, 128, 64), (4, 32, 48), (2, 9, 37), (1, 130, 7), (2, 80, 144), (1, 160, 256), (1, 1, 1)]


@pytest.mark.parametrize("H, D, V", MEMORY_SIZES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_memory_portions_and_single_tokens(dtype, H, D, V):
    """Four requests in slots out of order: portions on both sides of the chunks' borders beside single tokens, steps of
    single tokens in between, one request that sits steps out; outputs and states after every step."""
    mem = _Memories(H, D, V, dtype, seed=H * 100 + D)
    for s in range(4):
        mem.fresh(s)
    for i, (lens, slots) in enumerate([([2, 63, 1], [3, 0, 2]), ([1, 1, 1], [0, 3, 1]), ([64, 1], [1, 0]), ([65, 130, 2, 5], [2, 3, 0, 1]),
                                       ([1, 1, 1, 1], [1, 2, 0, 3]), ([127], [0]), ([1], [0]), ([3, 2], [0, 2])]):
        got, want = mem.step(lens, slots)
        _close(got, want, dtype, f"step {i}")
        mem.check_states(2e-5 if dtype == torch.float32 else 3e-4)


@pytest.mark.parametrize("shift", [(0.0, 0.0), (30.0, -30.0), (-30.0, 30.0), (30.0, 30.0), (-30.0, -30.0), (0.0, -8.0)])
@pytest.mark.parametrize("H, D, V", [(2, 64, 64), (2, 12, 10)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_memory_at_extreme_gates(dtype, H, D, V, shift):
    """Gates at their caps - sums of log forget gates of many hundreds within a chunk, inputs that vanish or outweigh
    everything - in portions and then in single tokens."""
    mem = _Memories(H, D, V, dtype, cap=15.0, seed=int(shift[0] * 7 + shift[1]) + D)
    mem.fresh(1)
    mem.fresh(2)
    for lens in ([200, 64], [1, 1], [70, 2], [1, 1]):
        got, want = mem.step(lens, [2, 1], gate_shift=shift)
        _close(got, want, dtype, str(lens))
    mem.check_states(5e-5 if dtype == torch.float32 else 3e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_memory_over_many_chunks_and_a_slot_used_again(dtype):
    """More chunks than the scan works on at a time (32), then the slot starts anew."""
    mem = _Memories(1, 16, 16, dtype, seed=5)
    mem.fresh(0)
    mem.fresh(3)
    got, want = mem.step([2300, 70], [0, 3])
    _close(got, want, dtype)
    mem.check_states(5e-5 if dtype == torch.float32 else 3e-4)
    mem.fresh(0)
    got, want = mem.step([5, 40], [3, 0])
    _close(got, want, dtype)
    got, want = mem.step([1, 1], [0, 3])
    _close(got, want, dtype)


def test_memory_is_the_same_however_it_is_cut():
    """FP32: one portion of 150 tokens, portions of many sizes, and single tokens leave the same outputs and state."""
    outs = []
    for cuts in ([150], [1, 63, 2, 64, 20], [2] * 75, [1] * 150):
        mem = _Memories(2, 24, 20, torch.float32, seed=9)
        mem.fresh(0)
        g = torch.Generator().manual_seed(1)
        H, D, V = 2, 24, 20
        proj, z = _rand(g, 150, 2 * H * (D + V)).to(DEV), _rand(g, 150, 2 * H, scale=2.0).to(DEV)
        ys, at = [], 0
        for n in cuts:
            y = torch.empty(n, H * V, device=DEV)
            common = (proj[at:at + n].contiguous(), z[at:at + n].contiguous(), 0, H, mem.bias_i.to(DEV), mem.bias_f.to(DEV), 9.0, mem.state,
                      torch.tensor([0, n], **I32), torch.tensor([0], **I32), 1)
            rest = (D ** -0.5, mem.weight.to(DEV), 1e-5)
            if n == 1:
                mem.ops.mlstm_token_step(*common, *rest, y, H, D, V)
            else:
                buf = torch.empty(mem.ops.mlstm_buffer_floats(n, 1, H, D, V), device=DEV)
                mem.ops.mlstm_chunk_step(*common, n, *rest, buf, torch.empty_like(y), y, H, D, V)
            ys.append(y)
            at += n
        outs.append((torch.cat(ys), mem.state[0].clone()))
    for y, st in outs[1:]:
        torch.testing.assert_close(y, outs[0][0], rtol=2e-4, atol=2e-5)
        torch.testing.assert_close(st, outs[0][1], rtol=1e-4, atol=2e-5)


# ---- differential attention ---------------------------------------------------------------------------------------

def _paged(g, lens, starts, G, kdim, vdim, page, dtype):
    """Cached keys and values of requests with ``starts`` tokens before this step's ``lens``, in pages out of order."""
    kv = [s + n for s, n in zip(starts, lens)]
    n_pages = sum(-(-k // page) for k in kv) + 3
    order = iter(torch.randperm(n_pages, generator=g).tolist())
    table = torch.zeros(len(lens), max(-(-k // page) for k in kv), dtype=torch.int32)
    kp, vp = torch.zeros(n_pages, G, page, kdim, dtype=dtype), torch.zeros(n_pages, G, page, vdim, dtype=dtype)
    K, V = [], []
    for s, n in enumerate(kv):
        K.append(_rand(g, n, G, kdim).to(dtype))
        V.append(_rand(g, n, G, vdim).to(dtype))
        for j in range(-(-n // page)):
            p = table[s, j] = next(order)
            m = min(page, n - j * page)
            kp[p, :, :m], vp[p, :, :m] = K[s][j * page:j * page + m].transpose(0, 1), V[s][j * page:j * page + m].transpose(0, 1)
    return K, V, kp.to(DEV), vp.to(DEV), table.to(DEV)


def _difference(q, K, V, lens, starts, H, G, D, scale, lam, eps, factor):
    n, vdim = q.shape[0], V[0].shape[-1]
    want, at = torch.zeros(n, H, vdim, dtype=F64), 0
    for s, ln in enumerate(lens):
        seen = torch.arange(starts[s] + ln)[None] <= (starts[s] + torch.arange(ln))[:, None]
        for h in range(H):
            g = h // (H // G)
            maps = [torch.softmax(((q[at:at + ln, h, m].double() @ K[s][:, g, m * D:(m + 1) * D].double().T) * scale)
                                  .masked_fill(~seen, float("-inf")), -1) @ V[s][:, g].double() for m in (0, 1)]
            u = maps[0] - lam * maps[1]
            want[at:at + ln, h] = u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps) * factor
        at += ln
    return want.view(n, H * vdim)


CASES = [([130, 17], [0, 40], 16), ([1, 2, 1], [500, 14, 15], 16), ([1, 140, 2], [200, 31, 0], 16), ([64, 5, 256], [0, 3, 129], 64),
         ([1, 1, 1, 1], [0, 127, 128, 900], 8), ([3], [0], 128)]


@pytest.mark.parametrize("lens, starts, page", CASES)
@pytest.mark.parametrize("H, G, D", [(4, 2, 64), (3, 1, 32), (4, 4, 64), (20, 1, 64), (16, 2, 32)])
def test_difference_in_the_tensor_core_kernels(H, G, D, lens, starts, page):
    """Both kernels against the equations and, position by position, against the plain kernel: single tokens in one to many
    splits, merged in a cluster and through scratch; heads that share a key head in groups of more than eight; portions
    whose rows end inside a tile."""
    from nanoinfer_b200.engine.step import upload_plans
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.mixer import DifferentialAttention, PagedAttendMixin
    g = torch.Generator().manual_seed(H * 100 + D + len(lens))
    bf, hd, n = torch.bfloat16, 2 * D, sum(lens)
    K, V, kp, vp, table = _paged(g, lens, starts, G, hd, hd, page, bf)
    q = _rand(g, n, H, 2, D, scale=1.5).to(bf)
    finish = (D ** -0.5, 0.43, 1e-6, 0.37)
    want = _difference(q, K, V, lens, starts, H, G, D, *finish)
    qd = q.view(n, -1).to(DEV)
    pos = torch.cat([torch.arange(s, s + x) for s, x in zip(starts, lens)]).to(**I32)
    seq = torch.repeat_interleave(torch.arange(len(lens)), torch.tensor(lens)).to(**I32)
    cu, kvl = torch.tensor([0] + list(torch.cumsum(torch.tensor(lens), 0)), **I32), torch.tensor([a + b for a, b in zip(starts, lens)], **I32)
    maps = torch.empty(n, 2 * H, hd, device=DEV)
    plain = torch.empty(n, H * hd, dtype=bf, device=DEV)
    ops.attention_generic(qd, kp, vp, maps.view(n, -1), pos, seq, table, 2 * H, G, D, page, None, finish[0], value_dim=hd, maps=2)
    ops.difference_norm(maps, plain, *finish[1:])
    torch.testing.assert_close(plain.cpu().double(), want, rtol=1e-2, atol=4e-3)
    plan = list(upload_plans([object.__new__(DifferentialAttention)], lens, starts, DEV).values())[0]
    out = torch.full_like(plain, float("nan"))
    if plan.scalars["n_tiles"]:
        ops.attention_prefill_difference(qd, kp, vp, out, plan.arrays["tile_seq"], plan.arrays["tile_row0"], plan.scalars["n_tiles"],
                                         cu, kvl, table, H, G, hd, page, *finish)
    dec = plan.arrays["dec_tokens"] if max(lens) > 1 else None
    n_dec, per = plan.scalars["n_dec"], H // G
    share = next(x for x in range(1, per + 1) if per % x == 0 and per // x <= 8)
    for splits, cluster in ((1, True), (3, True), (3, False), (11, False)) if n_dec else ((0, True),):
        if n_dec:
            scratch = torch.empty(n_dec * 2 * H * splits * (hd + 2), device=DEV)
            tickets = torch.zeros(n_dec * G * share, **I32)
            ops.attention_decode_cluster_merge(cluster)
            try:
                ops.attention_decode_difference(qd, kp, vp, out, dec, n_dec, pos, seq, table, H, G * share, hd, page, *finish, splits,
                                                scratch, tickets, share=share)
            finally:
                ops.attention_decode_cluster_merge(True)
            assert int(tickets.abs().sum()) == 0
        ops.check_device_errors(DEV)
        torch.testing.assert_close(out.cpu().double(), want, rtol=1.5e-2, atol=6e-3)


@pytest.mark.parametrize("H, G, D, V", [(4, 2, 24, 40), (3, 3, 9, 7), (2, 1, 40, 80), (1, 1, 130, 300)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_difference_in_the_plain_kernel(dtype, H, G, D, V):
    from nanoinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(D)
    lens, starts, page = [40, 1, 7], [3, 60, 14], 16
    n = sum(lens)
    K, Vs, kp, vp, table = _paged(g, lens, starts, G, 2 * D, V, page, dtype)
    q = _rand(g, n, H, 2, D).to(dtype)
    want = _difference(q, K, Vs, lens, starts, H, G, D, 0.3, 0.6, 1e-5, 0.8)
    pos = torch.cat([torch.arange(s, s + x) for s, x in zip(starts, lens)]).to(**I32)
    seq = torch.repeat_interleave(torch.arange(3), torch.tensor(lens)).to(**I32)
    maps, out = torch.empty(n, 2 * H, V, device=DEV), torch.zeros(n, H * V, dtype=dtype, device=DEV)
    for tokens in (torch.arange(0, 41), torch.arange(41, n)):              # a token list at a time
        tl = tokens.to(**I32)
        ops.attention_generic(q.view(n, -1).to(DEV), kp, vp, maps.view(n, -1), pos, seq, table, 2 * H, G, D, page, None, 0.3,
                              token_list=tl, value_dim=V, maps=2)
        ops.difference_norm(maps, out, 0.6, 1e-5, 0.8, token_list=tl)
    torch.testing.assert_close(out.cpu().double(), want, **(dict(rtol=2e-4, atol=2e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=4e-3)))


# ---- the routed feed-forward -----------------------------------------------------------------------------------------

@pytest.mark.parametrize("n", [1, 3, 8, 40, 700])
@pytest.mark.parametrize("E, top, groups, keep, scale", [(14, 4, 7, 3, 1.8), (8, 2, 4, 1, 1.3), (6, 6, 1, 1, 0.7), (5, 1, 5, 2, 1.0), (256, 40, 8, 3, 1.5)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_router_with_groups(dtype, E, top, groups, keep, scale, n):
    """The chosen experts (close calls aside), their weights over their sum times the factor, and the counts."""
    from nanoinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(E * 10 + n)
    d = 72
    x, w = _rand(g, n, d).to(dtype), _rand(g, E, d, scale=0.3)
    ids, wts, counts = torch.empty(n, top, **I32), torch.empty(n, top, device=DEV), torch.zeros(E, **I32)
    ops.route(x.to(DEV), w.to(DEV), None, ids, wts, counts, E, top, renormalize=True, groups=groups, keep_groups=keep, weight_scale=scale)
    assert torch.equal(torch.bincount(ids.view(-1).long().cpu(), minlength=E), counts.long().cpu())
    r = {"top": top, "scale": scale, "groups": {"count": groups, "keep": keep} if groups > 1 else None}
    same = 0
    for t in range(n):
        want_ids, want_w = choose_experts(w.double() @ x[t].double(), r)
        if ids[t].tolist() == want_ids:
            same += 1
            torch.testing.assert_close(wts[t].cpu().double(), torch.stack(want_w), rtol=2e-5, atol=1e-6)
    assert same >= n - max(1 if top > 8 else 0, n // 50)


@pytest.mark.parametrize("d", [1024, 1026, 2560, 2568, 5640, 12000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_router_at_other_widths(dtype, d):
    """Many tokens at widths that put eight, four and one of them into a block: the same choices and, bit for bit, the same
    weights as a few tokens at a time."""
    from nanoinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    n, E, top = 530, 17, 3
    x, w = _rand(g, n, d).to(dtype).to(DEV), _rand(g, E, d, scale=2.0 * d ** -0.5).to(DEV)

    def run(rows):
        ids, wts = torch.empty(rows.shape[0], top, **I32), torch.empty(rows.shape[0], top, device=DEV)
        ops.route(rows, w, None, ids, wts, None, E, top, renormalize=True)
        return ids, wts

    many = run(x)
    few = [run(x[a:a + 53].contiguous()) for a in range(0, n, 53)]
    assert torch.equal(many[0], torch.cat([f[0] for f in few])) and torch.equal(many[1], torch.cat([f[1] for f in few]))
    z = x.double() @ w.double().T
    want = torch.topk(torch.softmax(z, 1), top).values
    torch.testing.assert_close(many[1].double(), want / want.sum(1, keepdim=True), rtol=2e-4, atol=1e-6)


@pytest.mark.parametrize("E, top, F, d", [(10, 3, 88, 128), (8, 2, 40, 96), (6, 4, 20, 76), (1, 1, 16, 64)])
@pytest.mark.parametrize("n", [1, 4, 8, 20, 90])
@pytest.mark.parametrize("dtype", DTYPES)
def test_squared_relu_experts(dtype, n, E, top, F, d):
    """Every way the part multiplies with its experts (all of them for a few rows, pair by pair, laid out expert by
    expert), summed by itself and handed over as rows."""
    from nanoinfer_b200.config.model_config import FeedForwardSpec
    from nanoinfer_b200.engine.runtime import Runtime
    from nanoinfer_b200.parts.feed_forward import RoutedExperts
    g = torch.Generator().manual_seed(n * 100 + F)
    rt = Runtime(device=torch.device(DEV), dtype=dtype, page_size=16)
    groups = 2 if E % 2 == 0 and E // 2 >= top else 1
    spec = FeedForwardSpec(kind="routed_experts", intermediate_size=F,
                           extra=(("experts", E), ("top", top), ("unit", "relu2"), ("renormalize", True), ("weight_scale", 1.6), ("groups", groups), ("keep_groups", 1)))
    w = {"router": _rand(g, E, d, scale=0.4).to(dtype)}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = _rand(g, F, d, scale=d ** -0.5).to(dtype), _rand(g, d, F, scale=F ** -0.5).to(dtype)
    ffn = RoutedExperts(spec, d, w, rt)
    assert ffn.leaves_rows
    x = _rand(g, n, d).to(dtype)
    y = ffn.forward(x.to(DEV), None).cpu().double()
    left = ffn.forward(x.to(DEV), None, leave_rows=True)
    where = left.row_of_pair.view(n, top).long() if left.row_of_pair is not None else torch.arange(n * top, device=DEV).view(n, top)
    if left.all_experts:
        where = torch.arange(n, device=DEV)[:, None] * left.all_experts + left.ids.long()
    torch.testing.assert_close((left.weights.double()[..., None] * left.z.double()[where]).sum(1).cpu(), y, rtol=1e-4, atol=1e-5)
    wd = {k: v.double() for k, v in w.items()}
    mlp = {"router": {"top": top, "scale": 1.6, "groups": {"count": groups, "keep": 1} if groups > 1 else None}}
    want = torch.stack([pk.routed_unit(wd, "", mlp, x[t].double()) for t in range(n)])
    if dtype == torch.float32:
        torch.testing.assert_close(y, want, rtol=1e-4, atol=1e-5)
    else:                                                     # squares of rounded numbers: relative to the largest and to the whole
        err = (y - want).abs()
        assert err.max() <= 0.03 * want.abs().max() and err.pow(2).mean().sqrt() <= 0.01 * want.pow(2).mean().sqrt()


# ---- one layer, one token that counts ---------------------------------------------------------------------------------

def _runner(model_dir, dtype, steps, page=16, max_requests=4, **kw):
    from nanoinfer_b200.config import load_config
    from nanoinfer_b200.engine import ModelRunner
    from nanoinfer_b200.weights import load_weights
    cfg = load_config(model_dir)
    num_pages = max(1, ru.max_live_tokens(steps, 64) // page)
    return ModelRunner(cfg, load_weights(model_dir, cfg), dtype=dtype, page_size=page, num_pages=num_pages,
                       max_requests=max_requests, **kw)


def _follow(model_dir, dtype, prompts, want, cuts):
    """Feed each prompt in the portions that ``cuts`` names; the last logits against the plain ones."""
    from nanoinfer_b200.engine import StepEntry
    n = len(prompts["same"])
    runner = _runner(model_dir, dtype, ru.whole(prompts), max_requests=2)
    for k, toks in prompts.items():
        for a, b in zip(cuts, cuts[1:]):
            logits = runner.step([StepEntry(k, toks[a:b], [b - a - 1])])
        runner.end(k)
        ru.compare({(k, n - 1): logits[0].cpu()}, {k: {n - 1: want[k]}}, dtype, label=f"one token that counts, {k}")


FAR_CUTS = {"decoded": [0, 63, 64, 129, 250, 256, 257, 272, 290] + list(range(291, 301)), "prompt": [0, 2, 15, 17, 33, 160, 300],
            "short": [0, 128, 296, 298, 300]}


@pytest.mark.parametrize("kind", list(FAR_CUTS))
@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("D, V", [(24, 40), (32, 64), (64, 128)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_finds_a_far_key(tmp_path, dtype, D, V, shared, kind):
    """Token 4's query points - in the first map only - where token 2's key points (one coordinate of the embedding each,
    which no other token has), and nobody else's.  The prompt ends with token 4; token 2 stands only at position 3, hundreds
    of keys back.  ``shared``: the layer that looks back reads the keys and values of the layer before it."""
    last = 1 if shared else 0
    layers = [tk.attention(2, 1, D, V, 1.0, 0.4, None)] + ([tk.attention(2, 1, D, V, 1.0, 0.4, None, kv_from=0)] if shared else [])

    def more(t):
        e = t["embed"]
        e[:, 60:62] = 0
        e[2, 60] = 3.0                                   # what only token 2 has: most of its key
        e[4, 61] = 3.0                                   # what only token 4 has: most of its query
        for i in range(len(layers)):
            for n in (f"l{i}.norm1", f"l{i}.norm1.b"):
                t[n][60:62] = 1.0 if n.endswith("norm1") else 0.0
            t[f"l{i}.mix.q"][:, 60:62] = 0
        k = t["l0.mix.k"]
        k[:, 60], k[:, 61] = k[:, 60].sign() * 0.6, 0
        q = t[f"l{last}.mix.q"].view(2, 2, D, -1)
        q[:, 0, :, 61] = k[:D, 60] * (1.5 if D >= 32 else 2.0)
        if shared:
            t["l0.mix.o"].mul_(0.2)                      # (the two coordinates reach the second layer as they are)
            t["l0.mix.o"][60:62] = 0
        t[f"l{last}.mix.o"].mul_(4.0)
    raw = tk.model(120, 64, 2, layers)
    d = str(tmp_path / "m")
    tk.write_model(d, raw, 7, more=more)
    cfg, w = load_plain(d)
    n, far = 300, 3
    base = [5 + (i % 90) for i in range(n)]
    base[far], base[-1] = 2, 4
    other = list(base)
    other[far] = 3
    want = {k: whole_sequence(cfg, w, t)[-1].float() for k, t in (("same", base), ("other", other))}
    assert (want["same"] - want["other"]).abs().max().item() > 0.2 * want["same"].abs().max().item()
    _follow(d, dtype, {"same": base, "other": other}, want, FAR_CUTS[kind])


@pytest.mark.parametrize("kind", list(FAR_CUTS))
@pytest.mark.parametrize("H, D, V", [(2, 20, 12), (1, 64, 128)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_memory_keeps_a_far_token(tmp_path, dtype, H, D, V, kind):
    """Forget gates all but open, and an input gate that opens for token 2 alone: what it wrote at position 3 is still most
    of what the end reads 296 tokens later, through portions that end at and around chunk borders, then token by token."""
    def more(t):
        e = t["embed"]
        e[:, 60], e[:, 61] = -0.6, 0.0
        e[2, 60] = e[4, 61] = 3.0
        t["l0.norm1"][60:62], t["l0.norm1.b"][60:62] = 1.0, 0.0
        k, q = t["l0.mix.k"], t["l0.mix.q"]
        k[:, 60], k[:, 61] = k[:, 60].sign() * 0.6, 0.0
        q[:, 60], q[:, 61] = 0.0, k[:, 60] * 2.0             # the last token, 4, asks for what token 2 has left
        t["l0.mix.f"].zero_()
        t["l0.mix.f.b"].fill_(11.0)
        t["l0.mix.i"].mul_(0.1)
        t["l0.mix.i"][:, 60] = 6.0
        t["l0.mix.o"].mul_(6.0)
    raw = tk.model(120, 64, 2, [tk.memory(H, D, V, 14.0, None)])
    d = str(tmp_path / "m")
    tk.write_model(d, raw, H * D, more=more)
    cfg, w = load_plain(d)
    n, far = 300, 3
    base = [5 + (7 * i) % 90 for i in range(n)]
    base[far], base[-1] = 2, 4
    other = list(base)
    other[far] = 3
    want = {k: whole_sequence(cfg, w, t)[-1].float() for k, t in (("same", base), ("other", other))}
    assert (want["same"] - want["other"]).abs().max().item() > 0.2 * want["same"].abs().max().item()
    _follow(d, dtype, {"same": base, "other": other}, want, FAR_CUTS[kind])


# ---- whole models -----------------------------------------------------------------------------------------------------

CUTS = {"whole": ru.whole, "tail": ru.tail_by_token, "ragged": ru.ragged, "mixed": ru.mixed}
# lengths on both sides of the recurrence's chunk of 64 tokens and of pages of 16
LENGTHS = {"u1": [1, 2, 17, 64, 65, 130, 49], "u2": [3, 16, 63, 150, 31, 128], "u3": [2, 48, 66, 15, 33], "u4": [5, 1, 129, 23, 90]}
RAW = {"u1": tk.U1, "u2": tk.U2, "u3": tk.U3, "u4": tk.U4}
CLOSE_CALL = 0.05      # a gap between a router's logits below which bfloat16 roundings may turn a choice over


def _choice_gap(z, r):
    """How far a router's choice is from another one: the smaller of the gaps at the border of the chosen groups and at
    the border of the chosen experts (inf where there is no choice)."""
    gap, allowed = float("inf"), torch.ones_like(z, dtype=torch.bool)
    if r.get("groups") and r["groups"]["keep"] < r["groups"]["count"]:
        count, keep = r["groups"]["count"], r["groups"]["keep"]
        each = z.view(count, -1).max(1).values
        best = torch.sort(each, descending=True).values
        gap = (best[keep - 1] - best[keep]).item()
        allowed = torch.repeat_interleave(each >= best[keep - 1], z.numel() // count)
    left = torch.sort(z[allowed], descending=True).values
    if r["top"] < left.numel():
        gap = min(gap, (left[r["top"] - 1] - left[r["top"]]).item())
    return gap


def _with_gaps(cfg, w, toks, monkeypatch):
    """Plain logits [T, vocab] and every position's smallest choice gap."""
    orig, gaps = pk.choose_experts, [float("inf")]

    def watched(z, r):
        gaps[-1] = min(gaps[-1], _choice_gap(z, r))
        return orig(z, r)

    monkeypatch.setattr(pk, "choose_experts", watched)
    plain = PlainKepusun(cfg, w)
    st, rows = plain.new_state(), []
    for t in toks:
        rows.append(plain.token(int(t), st))
        gaps.append(float("inf"))
    monkeypatch.setattr(pk, "choose_experts", orig)
    return torch.stack(rows), gaps[:-1]


class _Positions:
    """What a comparison must know of single positions: ``close`` - those at which a router's choice is a close call -, and
    ``factor(rid, pos)`` >= 1 - how much more than the median position the logits there move when every weight is
    disturbed at the size of a bfloat16 rounding (a head's read-out that almost vanishes is magnified by its norm)."""

    def __init__(self, close=(), factors=None, names=None):
        self.close, self.factors, self.names = set(close), factors or {}, names or {}

    def is_close(self, rid, pos):
        return (self.names.get(rid, rid), pos) in self.close

    def factor(self, rid, pos):
        return self.factors.get((self.names.get(rid, rid), pos), 1.0)

    def renamed(self, names):
        return _Positions(self.close, self.factors, names)


def _sensitivity(cfg, w, reqs, want):
    g = torch.Generator().manual_seed(0)
    moved = {}
    for _ in range(2):
        shaken = {k: v.double() * (1 + 2.0 ** -12 * (torch.rand(v.shape, generator=g, dtype=F64) - 0.5)) for k, v in w.items()}
        for rid, toks in reqs.items():
            out = whole_sequence(cfg, shaken, toks).float()
            rel = (out - want[rid]).pow(2).mean(1).sqrt() / want[rid].pow(2).mean(1).sqrt()
            for pos in range(len(toks)):
                moved[(rid, pos)] = max(moved.get((rid, pos), 0.0), rel[pos].item())
    median = sorted(moved.values())[len(moved) // 2]
    return {k: max(1.0, v / (2.0 * median)) for k, v in moved.items()}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """{key: (folder, config dictionary, requests, plain logits per request, _Positions)}"""
    root = tmp_path_factory.mktemp("kepusun")
    mp = pytest.MonkeyPatch()
    out = {}
    for seed, (key, raw) in enumerate(RAW.items()):
        d = str(root / key)
        tk.write_model(d, raw, seed + 71)
        cfg, w = load_plain(d)
        reqs = {f"q{i}": random_tokens(raw["vocab"], n, 59 * seed + i) for i, n in enumerate(LENGTHS[key])}
        want, close = {}, set()
        for rid, toks in reqs.items():
            logits, gaps = _with_gaps(cfg, w, toks, mp)
            want[rid] = logits.float()
            close |= {(rid, p) for p, gap in enumerate(gaps) if gap < CLOSE_CALL}
        assert len(close) <= 0.4 * sum(LENGTHS[key]), f"{key}: too many close calls ({len(close)}): the test would cover little"
        out[key] = (d, cfg, reqs, want, _Positions(close, _sensitivity(cfg, w, reqs, want)))
    return out


# float32: the bounds of the Llama replays, the absolute one times the position's factor.  bfloat16: per position twice the
# bounds of the Llama replays times the factor; at most 3 % of the positions over them and none over four times.  Positions
# at which a router's choice is a close call are left out in bfloat16 (another expert may be chosen there; the 32-bit
# replays compare every position), and the three positions after one, whose mixers read what that token left, count among
# the 3 % but not for the worst.
BF16_MAX_REL, BF16_RMS_REL, BF16_SHARE_OVER, BF16_WORST = 0.10, 0.03, 0.03, 4.0


def _compare(got, want, dtype, label, at=_Positions()):
    ratios = {}
    for (rid, pos), row in got.items():
        ref, factor = want[rid][pos], at.factor(rid, pos)
        if dtype == "float32":
            torch.testing.assert_close(row, ref, rtol=ru.F32_RTOL, atol=ru.F32_ATOL * factor * max(1.0, ref.abs().max().item()),
                                       msg=lambda m: f"{label} request {rid} position {pos} (factor {factor:.1f}): {m}")
        elif not at.is_close(rid, pos):
            err = (row - ref).abs()
            ratios[(rid, pos)] = max(err.max().item() / (BF16_MAX_REL * factor * ref.abs().max().item()),
                                     err.pow(2).mean().sqrt().item() / (BF16_RMS_REL * factor * ref.pow(2).mean().sqrt().item()))
    if dtype == "float32":
        return
    assert ratios
    over = {k: round(v, 2) for k, v in ratios.items() if v > 1.0}
    worst = max([v for (rid, pos), v in ratios.items() if not any(at.is_close(rid, pos - b) for b in (1, 2, 3))] or [0.0])
    assert worst <= BF16_WORST, f"{label}: worst position at {worst:.2f} times the bound: {over}"
    assert len(over) <= max(1, BF16_SHARE_OVER * len(ratios)), f"{label}: {len(over)} of {len(ratios)} positions over the bound: {over}"


@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", list(RAW))
def test_replay_matches_plain(models, key, dtype, cut):
    """Exactly as many pages as the trace needs and four slots, so both are used again."""
    d, cfg, reqs, want, at = models[key]
    steps = CUTS[cut](reqs)
    runner = _runner(d, dtype, steps)
    got = ru.run_trace(runner, steps)
    assert len(got) == sum(len(t) for t in reqs.values())
    _compare(got, want, dtype, f"{key} {cut}", at)
    runner.cache.check_consistency()
    assert runner.cache.num_free_slots == 4


@pytest.mark.parametrize("page", [8, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_page_sizes(models, dtype, page):
    d, cfg, reqs, want, at = models["u2"]
    steps = ru.mixed(reqs, seed=3)
    _compare(ru.run_trace(_runner(d, dtype, steps, page=page), steps), want, dtype, f"pages of {page}", at)


@pytest.mark.parametrize("key", list(RAW))
def test_float32_barely_depends_on_the_cut(models, key):
    """In 32-bit the attention layers give the same bits under every cut; the recurrence sums a chunk's tokens in another
    order than token by token, so cuts may differ by FP32 roundings and no more."""
    d, cfg, reqs, want, at = models[key]
    ref = None
    for cut in CUTS:
        steps = CUTS[cut](reqs)
        got = ru.run_trace(_runner(d, "float32", steps), steps)
        if ref is None:
            ref = got
        for k in ref:
            scale = max(1.0, ref[k].abs().max().item())
            assert (ref[k] - got[k]).abs().max().item() <= 2e-5 * at.factor(*k) * scale, f"{key}: {cut} differs from whole at {k}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_short_portions(models, dtype):
    """Portions of two tokens from the sequence's start on, next to a request that starts with a single token."""
    d, cfg, reqs, want, at = models["u1"]
    a, b = reqs["q3"][:40], reqs["q4"][:21]
    steps = []
    for s, first in enumerate(range(0, 40, 2)):
        entries = [{"id": "a", "tokens": a[first:first + 2], "want": [0, 1]}]
        entries.append({"id": "b", "tokens": [b[s]], "want": [0]})
        steps.append({"step": s, "entries": entries, "end": []})
    got = ru.run_trace(_runner(d, dtype, steps), steps)
    _compare(got, {"a": want["q3"], "b": want["q4"]}, dtype, "short portions", at.renamed({"a": "q3", "b": "q4"}))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_replayed_graphs(models, dtype):
    """Most of a request token by token (the steps are captured and replayed from the third on), a second request decoding
    beside it from the middle on: 140 single-token steps move the recurrent states 140 times."""
    d, cfg, reqs, want, at = models["u2"]
    steps = ru.tail_by_token({"q3": reqs["q3"]}, tail=140)
    for i, st in enumerate(ru.tail_by_token({"q5": reqs["q5"]}, tail=60)):      # q5 runs beside q3's single tokens
        steps[30 + i]["entries"] += st["entries"]
        steps[30 + i]["end"] += st["end"]
    runner = _runner(d, dtype, steps)
    _compare(ru.run_trace(runner, steps), want, dtype, "long decoding", at)
    assert runner._graphs, "no step of single tokens was captured"


def test_recurring_portions_are_replayed(models):
    """The same portion size step after step is captured and replayed (bfloat16): states and caches move as before."""
    d, cfg, reqs, want, at = models["u2"]
    toks = reqs["q3"]
    steps = [{"step": i, "entries": [{"id": "q3", "tokens": toks[k:k + 10], "want": list(range(10))}], "end": []}
             for i, k in enumerate(range(0, 150, 10))]
    runner = _runner(d, "bfloat16", steps)
    _compare(ru.run_trace(runner, steps), want, "bfloat16", "recurring portions", at)
    assert runner._portion_graphs, "no recurring portion was captured"


def test_greedy_generation_through_the_engine(models):
    """Engine.generate (scheduler, chunked prompts, sampling kernels) against greedy decoding of the plain model."""
    from nanoinfer_b200 import Engine, SamplingParams
    d, cfg, reqs, want, at = models["u1"]
    raw_cfg, w = load_plain(d)
    plain = PlainKepusun(raw_cfg, w)
    prompts = [reqs["q2"], reqs["q3"][:20], reqs["q6"], reqs["q1"]]
    engine = Engine.from_model_dir(d, dtype="float32", block_size=16, num_cache_blocks=64, max_batch_size=4,
                                   max_sequences=4, prefill_chunk_size=12)
    out = engine.generate(prompts, max_new_tokens=12, sampling_params=SamplingParams.greedy())
    for prompt, got in zip(prompts, out):
        st = plain.new_state()
        logits = plain.run(prompt, st)[-1]
        for t in got:
            if int(torch.argmax(logits)) != t:
                assert (logits.max() - logits[t]).item() < 1e-4, "the engine chose a token that the plain model ranks lower"
            logits = plain.run([t], st)[-1]
        assert len(got) == 12


def test_a_preempted_request_starts_from_an_empty_state(models):
    """Too few pages for all requests at once: the scheduler preempts and recomputes, and every token stays the same."""
    from nanoinfer_b200 import Engine, SamplingParams
    d, cfg, reqs, want, at = models["u1"]
    prompts = [reqs["q3"][:30], reqs["q4"][:31], reqs["q6"][:29]]
    tokens = {}
    for blocks in (64, 8):
        engine = Engine.from_model_dir(d, dtype="float32", block_size=16, num_cache_blocks=blocks, max_batch_size=3, max_sequences=3,
                                       prefill_chunk_size=16)
        engine.stop_token_ids = ()
        tokens[blocks] = engine.generate(prompts, max_new_tokens=24, sampling_params=SamplingParams.greedy())
        if blocks == 8:
            assert engine.get_scheduler_stats().num_preemptions > 0
    assert tokens[8] == tokens[64]


def test_trace_replay_from_the_command_line(models, tmp_path):
    """bin/trace_run as a user runs it: the model class follows from config.json."""
    d, cfg, reqs, want, at = models["u4"]
    reqs = {k: reqs[k] for k in ("q2", "q3")}
    steps = ru.mixed(reqs, tail=4)
    out = str(tmp_path / "out")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out,
                        "--max-tokens", str(ru.max_live_tokens(steps, 64))], input="\n".join(json.dumps(s) for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    got, fed = {}, {}
    for st in steps:
        n_want = sum(len(e["want"]) for e in st["entries"])
        rows = torch.from_file(os.path.join(out, f"{st['step']}.f32"), size=n_want * cfg["vocab"], dtype=torch.float32).view(n_want, -1)
        r = 0
        for e in st["entries"]:
            for wpos in e["want"]:
                got[(e["id"], fed.get(e["id"], 0) + wpos)] = rows[r].clone()
                r += 1
            fed[e["id"]] = fed.get(e["id"], 0) + len(e["tokens"])
    _compare(got, want, "float32", "trace_run", at)
