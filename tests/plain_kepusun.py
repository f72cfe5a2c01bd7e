"""A plain, slow implementation of the Kepusun design in FP64: one function per mechanism, token by token, with Python
lists as caches.  It shares no code with the package and knows nothing of pages, slots or steps; the tests compare
the engine with it.

Notation: X is the list of streams, h a sublayer's input, w the dictionary of tensors by name.  Weights are [out, in]
and applied as W h.
"""
import math

import torch

F64 = torch.float64


def unit_rms(x, eps):
    """x divided by its root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean() + eps)


def dynamic_tanh(x, w, name):
    """tanh of the scaled input, times a weight, plus a bias, coordinate by coordinate: no statistics."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def read_streams(X, coef):
    """A sublayer's input before its norm: the streams weighted and summed."""
    return sum(coef[s] * x for s, x in enumerate(X))


def write_streams(X, mix, out, y):
    """Every stream anew from all the old ones (mix is indexed [from, to]), plus its share of the sublayer's output."""
    return [sum(mix[s, t] * X[s] for s in range(len(X))) + out[t] * y for t in range(len(X))]


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def value_size(m):
    """The size of a value: that of a key unless the mixer says otherwise."""
    return m["dim"] if m.get("vdim") is None else m["vdim"]


def fresh_memory(m):
    """[matrix [dim, vdim], normaliser [dim], running maximum] per head, all zero."""
    return [[torch.zeros(m["dim"], value_size(m), dtype=F64), torch.zeros(m["dim"], dtype=F64), torch.zeros((), dtype=F64)]
            for _ in range(m["heads"])]


def memory_step(mem, q, k, v, i_log, f_log):
    """One token of one head: the memory is rescaled to the new running maximum, takes the token, and is read.
    ``mem`` = [S, n, m] is changed in place."""
    S, n, m = mem
    top = torch.maximum(f_log + m, i_log)
    keep, take = torch.exp(f_log + m - top), torch.exp(i_log - top)
    S = keep * S + take * torch.outer(k, v)
    n = keep * n + take * k
    mem[:] = [S, n, top]
    return (S.T @ q) / (torch.maximum((n @ q).abs(), torch.exp(-top)) + 1e-6)


def memory_mixer(w, pre, m, h, mem, eps):
    """The matrix-memory mixer: exponential input gate, sigmoid forget gate, both logs capped; a norm per head, a
    weight over all heads, a sigmoid gate."""
    H, D, V, cap = m["heads"], m["dim"], value_size(m), m["gate_cap"]
    q, k, v = (w[pre + "q"] @ h).view(H, D) * D ** -0.5, (w[pre + "k"] @ h).view(H, D), (w[pre + "v"] @ h).view(H, V)
    i_log = capped(w[pre + "i"] @ h + w[pre + "i.b"], cap)
    f_log = torch.nn.functional.logsigmoid(capped(w[pre + "f"] @ h + w[pre + "f.b"], cap))
    outs = [unit_rms(memory_step(mem[a], q[a], k[a], v[a], i_log[a], f_log[a]), eps) for a in range(H)]
    return w[pre + "o"] @ (torch.cat(outs) * w[pre + "norm"] * torch.sigmoid(w[pre + "g"] @ h))


def softmax_read(scores, values):
    p = torch.softmax(scores, dim=0)
    return p @ values


def difference_weight(w, pre, diff):
    """How much of the second map is taken off the first: one number per layer."""
    return math.exp((w[pre + "lq1"] * w[pre + "lk1"]).sum().item()) - math.exp((w[pre + "lq2"] * w[pre + "lk2"]).sum().item()) + diff


def difference_attention(w, pre, m, h, cache, eps, own):
    """Two attention maps per head over the same values, the second taken off the first; the rest to unit root mean
    square, times 1 - diff.  ``cache`` is the list of (keys [G, 2, dim], values [G, vdim]) of the tokens so far; a
    layer with projections of its own (``own``) appends this token's."""
    H, D, V = m["heads"], m["dim"], value_size(m)
    G = H if m.get("kv_heads") is None else m["kv_heads"]
    q = (w[pre + "q"] @ h).view(H, 2, D)
    if own:
        cache.append(((w[pre + "k"] @ h).view(G, 2, D), (w[pre + "v"] @ h).view(G, V)))
    K, Vs = torch.stack([k for k, _ in cache]), torch.stack([v for _, v in cache])
    lam = difference_weight(w, pre, m["diff"])
    heads = []
    for a in range(H):
        g = a // (H // G)
        one, two = (softmax_read((K[:, g, i] @ q[a, i]) * m["scale"], Vs[:, g]) for i in (0, 1))
        heads.append(unit_rms(one - lam * two, eps) * (1.0 - m["diff"]))
    return w[pre + "o"] @ torch.cat(heads)


def choose_experts(z, r):
    """(numbers, weights) of the chosen experts for router logits z: softmax over all, the best groups by their best
    expert, the best experts in those, their scores over their sum, times a factor."""
    s = torch.softmax(z, dim=0)
    allowed = torch.ones_like(s, dtype=torch.bool)
    if r.get("groups"):
        count, keep = r["groups"]["count"], r["groups"]["keep"]
        best = s.view(count, -1).max(dim=1).values
        allowed[:] = False
        for g in torch.topk(best, keep).indices.tolist():
            allowed.view(count, -1)[g] = True
    ids = torch.topk(torch.where(allowed, s, torch.full_like(s, -1.0)), r["top"]).indices.tolist()
    total = sum(s[e] for e in ids) + 1e-20
    return ids, [s[e] / total * r["scale"] for e in ids]


def expert(w, pre, h):
    """One expert: up, the square of the positive part, down."""
    return w[pre + "down"] @ torch.relu(w[pre + "up"] @ h) ** 2


def routed_unit(w, pre, mlp, h):
    ids, weights = choose_experts(w[pre + "router"] @ h, mlp["router"])
    return sum(p * expert(w, f"{pre}e{e}.", h) for e, p in zip(ids, weights))


class PlainKepusun:
    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: v.to(F64) for k, v in weights.items()}
        self.eps = cfg["norm"]["eps"]

    def new_state(self):
        kept = []
        for layer in self.cfg["layers"]:
            m = layer["mixer"]
            kept.append(fresh_memory(m) if layer["type"] == "mlstm" else (None if m.get("kv_from") is not None else []))
        return {"layers": kept, "sums": []}

    def mixer(self, i, h, kept):
        layer, pre = self.cfg["layers"][i], f"l{i}.mix."
        m = layer["mixer"]
        if layer["type"] == "mlstm":
            return memory_mixer(self.w, pre, m, h, kept[i], self.eps)
        j = m.get("kv_from")
        return difference_attention(self.w, pre, m, h, kept[i if j is None else j], self.eps, j is None)

    def token(self, tok, st):
        """Logits after one more token of the sequence whose state is st; st["sums"] gets the sum of the streams after
        every layer."""
        w = self.w
        X = [w["embed"][tok]] * self.cfg["streams"]
        sums = []
        for i, layer in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            y = self.mixer(i, dynamic_tanh(read_streams(X, w[p + "hc1.in"]), w, p + "norm1"), st["layers"])
            X = write_streams(X, w[p + "hc1.mix"], w[p + "hc1.out"], y)
            if layer.get("mlp"):
                y = routed_unit(w, p + "mlp.", layer["mlp"], dynamic_tanh(read_streams(X, w[p + "hc2.in"]), w, p + "norm2"))
                X = write_streams(X, w[p + "hc2.mix"], w[p + "hc2.out"], y)
            sums.append(sum(X))
        st["sums"] = sums
        return w["head"] @ dynamic_tanh(sum(X), w, "final.norm")

    def run(self, tokens, st):
        return torch.stack([self.token(int(t), st) for t in tokens])


def whole_sequence(cfg, weights, tokens):
    """Logits [T, vocab] of one sequence from its start."""
    plain = PlainKepusun(cfg, weights)
    return plain.run(tokens, plain.new_state())
