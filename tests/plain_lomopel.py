"""A plain, slow implementation of the Lomopel design in FP64: one function per mechanism, Python lists as caches, one
token after the other.  It shares no code with the package and knows nothing of pages, slots or steps; the tests compare
the engine with it.

Notation: x is the stream, h a sublayer's normed input, w the dictionary of tensors by name.  Matrices are [out, in] and
applied as W h.
"""
import math

import torch

F64 = torch.float64


def unit_rms(x, eps):
    """x divided by its root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean() + eps)


def shifted_norm(x, weight, eps):
    """RMS norm whose stored weight lies around zero: the gain is 1 + weight."""
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    """The tanh form of gelu."""
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softmax_read(scores, values, sink=None):
    """sum_j p_j values_j with p the softmax of the scores; `sink` (a number): one more term exp(sink) in the denominator."""
    s = torch.stack(scores)
    top = s.max().item() if sink is None else max(s.max().item(), float(sink))
    e = torch.exp(s - top)
    total = e.sum() + (0.0 if sink is None else math.exp(float(sink) - top))
    return sum(p * v for p, v in zip(e / total, values))


def temperature(q_temp, pos):
    """The factor on the query at a position: it grows with the logarithm of how many stretches of `every` tokens have passed."""
    if not q_temp:
        return 1.0
    return 1.0 + q_temp["coef"] * math.log(math.floor((pos + 1) / q_temp["every"]) + 1)


def mixed_value(v, first, lam):
    """A layer's values and the first value-mixing layer's values of the same token, (1 - lam) : lam."""
    return (1.0 - lam) * v + lam * first


def attention_value(w, pre, m, h):
    """The layer's own values [G, V] of one token, before any mixing."""
    return (w[pre + "v"] @ h + w[pre + "v.b"]).view(m["kv_heads"], m["vdim"])


def sink_attention(w, pre, m, h, pos, cache, v, leave_out=None):
    """Causal attention without rotation: biased projections, a query factor that grows with the position, a learned sink
    per head, a biased output projection.  `v`: the token's values as they are cached."""
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (w[pre + "q"] @ h + w[pre + "q.b"]).view(H, D)
    k = (w[pre + "k"] @ h + w[pre + "k.b"]).view(G, D)
    if leave_out != "q_temp":
        q = q * temperature(m.get("q_temp"), pos)
    cache.append((k, v))
    heads = []
    for a in range(H):
        g = a // (H // G)
        sink = None if leave_out == "sink" else w[pre + "sink"][a]
        heads.append(softmax_read([(q[a] @ kk[g]) * m["scale"] for kk, _ in cache], [vv[g] for _, vv in cache], sink))
    return w[pre + "o"] @ torch.cat(heads) + w[pre + "o.b"]


def rotate(v, pos, rot):
    """Entries i and i + n/2 of the first n = rot.dims entries of v turned by pos * base^(-2i/n)."""
    n = rot["dims"] if rot else 0
    half = n // 2
    out = v.clone()
    for i in range(half):
        a = pos * rot["base"] ** (-2.0 * i / n)
        c, s = math.cos(a), math.sin(a)
        out[i] = v[i] * c - v[i + half] * s
        out[i + half] = v[i + half] * c + v[i] * s
    return out


def in_window(pos, j, size):
    return 0 <= pos - j and (size is None or pos - j < size)


def window_attention(w, pre, m, h, pos, cache, eps):
    """Rotated queries and keys, every head of both to unit root mean square; the last mask.size tokens; every coordinate
    of the result times a sigmoid gate of the input."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (w[pre + "q"] @ h).view(H, D), (w[pre + "k"] @ h).view(G, D), (w[pre + "v"] @ h).view(G, V)
    q = torch.stack([unit_rms(rotate(x, pos, m["rot"]), eps) for x in q])
    k = torch.stack([unit_rms(rotate(x, pos, m["rot"]), eps) for x in k])
    cache.append((k, v))
    size = m["mask"]["size"] if m.get("mask") else None
    seen = [j for j in range(pos + 1) if in_window(pos, j, size)]
    heads = []
    for a in range(H):
        g = a // (H // G)
        heads.append(softmax_read([(q[a] @ cache[j][0][g]) * m["scale"] for j in seen], [cache[j][1][g] for j in seen]))
    return w[pre + "o"] @ (torch.cat(heads) * torch.sigmoid(w[pre + "g"] @ h))


def convolved(x, taps, past):
    """silu of the causal convolution of one token's channels: `past` holds the inputs before it, the oldest first, and
    moves on by one; taps [channels, K], the last column for the token itself."""
    rows = past + [x]
    y = sum(taps[:, j] * r for j, r in enumerate(rows))
    past[:] = rows[1:]
    return silu(y)


def delta_state(m):
    G, H, D, V, K = m["kv_heads"], m["heads"], m["dim"], m["vdim"], m["conv"]
    zeros = lambda n: [torch.zeros(n, dtype=F64) for _ in range(K - 1)]      # noqa: E731
    return {"S": [torch.zeros(D, V, dtype=F64) for _ in range(H)], "q": zeros(G * D), "k": zeros(G * D), "v": zeros(H * V)}


def delta_step(S, g, beta, q, k, v):
    """One token of the rule for one head: the rows of S decay (g, one factor per row), the error of the state's answer
    to k is written back, and q reads the new state.  Returns (S, o)."""
    S = g[:, None] * S
    S = S + torch.outer(k, beta * (v - S.T @ k))
    return S, S.T @ q


def delta_mixer(w, pre, m, h, st, eps):
    """The gated delta rule with one decay per head and key channel, from a two-step projection, and an output gate from
    another one."""
    G, H, D, V = m["kv_heads"], m["heads"], m["dim"], m["vdim"]
    q = convolved(w[pre + "q"] @ h, w[pre + "q.conv"], st["q"]).view(G, D)
    k = convolved(w[pre + "k"] @ h, w[pre + "k.conv"], st["k"]).view(G, D)
    v = convolved(w[pre + "v"] @ h, w[pre + "v.conv"], st["v"]).view(H, V)
    beta = torch.sigmoid(w[pre + "b"] @ h)
    z = w[pre + "a2"] @ (w[pre + "a1"] @ h) + w[pre + "dt_bias"]
    decay = torch.exp(-torch.exp(w[pre + "A_log"])[:, None] * torch.nn.functional.softplus(z).view(H, D))
    outs = []
    for a in range(H):
        g = a // (H // G)
        kk = k[g] / torch.sqrt((k[g] * k[g]).sum() + 1e-6)
        qq = q[g] / torch.sqrt((q[g] * q[g]).sum() + 1e-6) * D ** -0.5
        st["S"][a], o = delta_step(st["S"][a], decay[a], beta[a], qq, kk, v[a])
        outs.append(unit_rms(o, eps) * w[pre + "norm"])
    return w[pre + "o"] @ (torch.cat(outs) * torch.sigmoid(w[pre + "g2"] @ (w[pre + "g1"] @ h)))


def gelu_unit(w, pre, h):
    return w[pre + "down"] @ (gelu_tanh(w[pre + "gate"] @ h) * (w[pre + "up"] @ h))


class PlainLomopel:
    def __init__(self, cfg, weights):
        self.cfg, self.eps = cfg, cfg["norm"]["eps"]
        self.w = {k: v.to(F64) for k, v in weights.items()}
        self.first_mixing = next((i for i, la in enumerate(cfg["layers"])
                                  if la["type"] == "attention" and la["mixer"].get("v_mix")), None)

    def new_state(self):
        return {"pos": 0, "layers": [[] if la["type"] == "attention" else ([], delta_state(la["mixer"]["right"]))
                                     for la in self.cfg["layers"]]}

    def mixer(self, i, h, pos, kept, shared, leave_out=None):
        layer, pre, w = self.cfg["layers"][i], f"l{i}.mix.", self.w
        m = layer["mixer"]
        if layer["type"] == "attention":
            v = attention_value(w, pre, m, h)
            if i == self.first_mixing:
                shared["v"] = v
            elif m.get("v_mix") and leave_out != "v_mix":
                v = mixed_value(v, shared["v"], w[pre + "vmix"])
            return sink_attention(w, pre, m, h, pos, kept, v, leave_out)
        left = window_attention(w, pre + "left.", m["left"], h, pos, kept[0], self.eps)
        right = delta_mixer(w, pre + "right.", m["right"], h, kept[1], self.eps)
        return m["left_scale"] * left + m["right_scale"] * right

    def token(self, tok, st, after=None, leave_out=None):
        """Logits after one more token of the sequence whose state is st; ``after`` (a list) receives the stream after
        every layer; ``leave_out``: a mechanism that is skipped (for tests that show it matters)."""
        w, pos = self.w, st["pos"]
        x = w["embed"][tok] * (1.0 if leave_out == "embedding_scale" else self.cfg["embedding"]["scale"])
        shared = {}
        for i, layer in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            y = self.mixer(i, shifted_norm(x, w[p + "norm1"], self.eps), pos, st["layers"][i], shared, leave_out)
            x = x + (y if leave_out == "ls1" else y * w[p + "ls1"])
            if layer.get("mlp"):
                y = gelu_unit(w, p + "mlp.", shifted_norm(x, w[p + "norm2"], self.eps))
                x = x + (y if leave_out == "ls2" else y * w[p + "ls2"])
            if after is not None:
                after.append(x)
        st["pos"] = pos + 1
        return w["head"] @ shifted_norm(x, w["final.norm"], self.eps)

    def run(self, tokens, st):
        return torch.stack([self.token(int(t), st) for t in tokens])


def whole_sequence(cfg, weights, tokens):
    """Logits [T, vocab] of one sequence from its start."""
    plain = PlainLomopel(cfg, weights)
    return plain.run(tokens, plain.new_state())
