"""Recurrent token mixers: a fixed-size state per request instead of a cache that grows."""
from __future__ import annotations

from typing import Dict

import torch

from ..config.model_config import ConfigError
from ..config.registry import part, register_part
from ..kernels import ops
from .base import FreeDim, Part, StateNeed, WeightSlot


class GatedDeltaRule(Part):
    """The gated delta rule.  Per value head, with a matrix state M [dim, value_dim] in FP32 - the token first predicts its own value from
    the decayed state, writes the error back under its key, and reads with its query what the state then holds:

        M *= decay;   e = beta * (v - k M);   M += outer(k, e);   y = q M      (k, q rows of size dim; v, e, y of size value_dim)

    q and k (``num_kv_heads`` heads of ``head_dim``; value head h reads head h / (heads / kv heads)) and
    v (``num_heads`` heads of ``value_dim``) pass a short causal convolution over time per channel
    (``conv_taps`` taps, the last one the current token's, no bias) and silu; q and k are then unit
    vectors per head (1e-6 under the root), q also times head_dim^-1/2.  beta = sigmoid(W_b x), one per
    head.  Each head's y is divided by its root mean square (``norm_eps``), multiplied by a weight [value_dim] shared by
    the heads and by a gate, and leaves through W_o.  Two options in the spec's extra:

    ``decay``  "head" (the default): one decay per head, exp(-exp(A_log) softplus(W_a x + dt_bias));
               "key_channel": one per head and key channel, exp(-exp(A_log_h) softplus(W_a2 (W_a1 x) + dt_bias)), which
               multiplies the rows of M - W_a1 and W_a2 are thin, their inner size follows from the stored tensors;
    ``gate``   "silu" (the default): silu(W_g x); "low_rank_sigmoid": sigmoid(W_g2 (W_g1 x)), thin in the same way.

    All projections of x are ONE product (rows q | k | v | gate | b | a, or q | k | v | b | a1 | g1); with thin matrices a
    second, block-diagonal product turns (W_a1 x, W_g1 x) into the logits of decay and gate in FP32.  Everything from there
    to the gated norm is FP32 on the device; in bfloat16 a step of single tokens with both options is one launch (from an
    FP32 projection, thin products included), and portions of CHUNK_FROM tokens and more run in chunks on the tensor cores
    (csrc/delta_chunk.cu).  A request's state is one FP32 vector: M of every head, then the last
    conv_taps - 1 inputs of every convolved channel.  A step's kernels run exactly once, so the state advances by exactly
    the step's tokens.

    ``joined`` in the extra: one side of mixers that share their input and output projections (ParallelMixers)."""

    kernel_modules = ("delta_rule",)       # libraries of csrc that this part's kernels live in

    CHUNK_FROM = 16             # a step whose longest portion has this many tokens takes the chunked recurrence

    JOINS = True                # can be a side of mixers with joined projections
    takes_output_scale = True   # a factor on the output rides in the gated norm, before the output projection
    output_scale = 1.0

    adds_into_residual = True
    graph_safe = "all"

    @staticmethod
    def _dims(spec):
        e = spec.extra_dict()
        return spec.num_kv_heads, spec.num_heads, spec.head_dim, int(e["value_dim"]), int(e["conv_taps"])

    @staticmethod
    def _options(spec):
        e = spec.extra_dict()
        decay, gate = e.get("decay", "head"), e.get("gate", "silu")
        if decay not in ("head", "key_channel") or gate not in ("silu", "low_rank_sigmoid"):
            raise ConfigError(f"gated delta rule: decay '{decay}' (head, key_channel) or gate '{gate}' (silu, low_rank_sigmoid) "
                              f"is not known")
        return decay == "key_channel", gate == "low_rank_sigmoid"

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        g, h, d, v, taps = GatedDeltaRule._dims(spec)
        channel, thin_gate = GatedDeltaRule._options(spec)
        slots = {"q": WeightSlot((g * d, hidden_size)), "q.conv": WeightSlot((g * d, taps)),
                 "k": WeightSlot((g * d, hidden_size)), "k.conv": WeightSlot((g * d, taps)),
                 "v": WeightSlot((h * v, hidden_size)), "v.conv": WeightSlot((h * v, taps)),
                 "b": WeightSlot((h, hidden_size)), "A_log": WeightSlot((h,)), "norm": WeightSlot((v,), init="ones")}
        if channel:
            rank = FreeDim(d, "decay_rank")
            slots.update({"a1": WeightSlot((rank, hidden_size)), "a2": WeightSlot((h * d, rank)), "dt_bias": WeightSlot((h * d,))})
        else:
            slots.update({"a": WeightSlot((h, hidden_size)), "dt_bias": WeightSlot((h,))})
        if thin_gate:
            rank = FreeDim(v, "gate_rank")
            slots.update({"g1": WeightSlot((rank, hidden_size)), "g2": WeightSlot((h * v, rank))})
        else:
            slots["g"] = WeightSlot((h * v, hidden_size))
        slots["o"] = WeightSlot((hidden_size, h * v))
        return slots

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        super().__init__(spec, hidden_size, weights, rt)
        g, h, d, v, taps = self._dims(spec)
        if g <= 0 or h <= 0 or h % g:
            raise ConfigError("gated delta rule: heads must be a positive multiple of kv_heads")
        if not 0 < d <= 1024:
            raise ConfigError(f"gated delta rule: a key size of {d} is not supported (1 to 1024)")
        if v <= 0 or taps <= 0:
            raise ConfigError("gated delta rule: value size and convolution taps must be positive")
        self.G, self.H, self.D, self.V, self.taps = g, h, d, v, taps
        self.channel, self.thin_gate = self._options(spec)
        self.eps = float(spec.extra_dict().get("norm_eps", 1e-6))
        self.channels = 2 * g * d + h * v
        rows = [weights[s] for s in ("q", "k", "v")]
        at = self.channels
        self.gate_col = at                                     # (a full gate's)
        if not self.thin_gate:
            rows.append(weights["g"])
            at += h * v
        self.b_col = at
        rows.append(weights["b"])
        at += h
        if not self.channel:
            rows.append(weights["a"])
            at += h
        joined = bool(spec.extra_dict().get("joined", False))
        like = weights["q"]

        def zeros(n, k):
            return torch.zeros(n, k, dtype=like.dtype, device=like.device)

        # the thin matrices: their inner sizes padded with zeros to multiples of 8, from a multiple of 8 columns on
        self.thin_col = self.thin_k = 0
        self.w_thin = None
        if self.channel or self.thin_gate:
            if at % 8:
                rows.append(zeros(-at % 8, hidden_size))
            self.thin_col = at + -at % 8
            pairs = ([("a1", "a2")] if self.channel else []) + ([("g1", "g2")] if self.thin_gate else [])
            second, self.ranks = [], {}
            for one, two in pairs:
                rank = weights[one].shape[0]
                if weights[two].shape[1] != rank:
                    raise ConfigError(f"gated delta rule: {one} and {two} differ in their inner size")
                rows += [weights[one]] + ([zeros(-rank % 8, hidden_size)] if rank % 8 else [])
                padded = torch.cat([weights[two], zeros(weights[two].shape[0], -rank % 8)], dim=1)
                second.append(padded)
                self.ranks[one] = padded.shape[1]
                self.thin_k += padded.shape[1]
            self.w_second = [rt.weight(x) for x in second]
            self.w_thin = rt.weight(torch.block_diag(*[x.float() for x in second]).to(like.dtype))        # [H D (+ H V), ranks]
            at = self.thin_col + self.thin_k
        if joined and at % 8:
            rows.append(zeros(-at % 8, hidden_size))
        if joined:
            self.in_rows, self.out_matrix = torch.cat(rows, dim=0), weights["o"]
        else:
            self.w_in = rt.weight(torch.cat(rows, dim=0))
            self.w_o = rt.weight(weights["o"])
        self.conv_w = rt.gain(torch.cat([weights[s] for s in ("q.conv", "k.conv", "v.conv")], dim=0))
        self.a_log, self.dt_bias = rt.gain(weights["A_log"]), rt.gain(weights["dt_bias"])
        self.norm_w = rt.gain(weights["norm"])
        # single tokens go through one kernel, which reads an FP32 projection
        self.wants_f32_tokens = (rt.dtype == torch.bfloat16 and self.channel and self.thin_gate
                                 and max(d, v) <= ops.DELTA_TOKEN_MAX_DIM and self.thin_k <= 8192)
        self.chunked = rt.dtype == torch.bfloat16 and self.channel and d <= ops.DELTA_CHUNK_MAX_DIM and v <= 512
        if self.chunked:
            self.kernel_modules = ("delta_chunk",)

    def cache_need(self):
        return StateNeed((self.H * self.D * self.V + (self.taps - 1) * self.channels,), "float32")

    def weights_in_order(self) -> tuple:
        return (self.w_in, self.w_o)

    def forward(self, x: torch.Tensor, ctx, cache, residual=None):
        dtype = self.rt.dtype if self._in_chunks(ctx) else torch.float32
        return self.finish(self.rt.linear(x, self.w_in, out_dtype=dtype), ctx, cache, residual=residual)

    def _in_chunks(self, ctx) -> bool:
        return self.chunked and ctx.max_q_len >= self.CHUNK_FROM

    def project(self, h: torch.Tensor, norm) -> torch.Tensor:
        """The fused input projection of norm(h), with the norm inside the product (steps of a few rows): the first
        half of forward for an arrangement that lets all its sublayers read the stream before any adds into it."""
        proj = self.rt.empty(h.shape[0], self.w_in.shape[0], dtype=torch.float32)
        ops.gemv_norm_bf16(h, norm.gain, norm.eps, None, self.w_in, proj, ops.STORE_F32)
        return proj

    def finish(self, proj: torch.Tensor, ctx, cache, residual=None):
        y = self.rt.empty(proj.shape[0], self.H * self.V)
        self.between(proj, 0, ctx, cache, out=y)
        return self.rt.linear(y, self.w_o, residual=residual)

    def _thin_logits(self, proj: torch.Tensor, col0: int):
        """FP32 [T, H D (+ H V)]: the logits of decay and gate from their thin first products in ``proj``."""
        rt = self.rt
        n = proj.shape[0]
        x = proj[:, col0 + self.thin_col:col0 + self.thin_col + self.thin_k]
        if rt.dtype == torch.float32:
            z = rt.empty(n, self.w_thin.shape[0])
            ops.gemm_f32_heads(x, self.w_thin.view(1, *self.w_thin.shape), z)
            return z
        if x.dtype != torch.bfloat16 or rt.skinny(n, self.thin_k):
            x = x.to(torch.bfloat16).contiguous()
        return rt.linear(x, self.w_thin, out_dtype=torch.float32)

    def between(self, proj: torch.Tensor, col0: int, ctx, cache, out: torch.Tensor, out_col: int = 0) -> torch.Tensor:
        """Everything between the projections: from columns ``col0`` on of proj to the gated, normed read-outs in columns
        ``out_col`` on of ``out``."""
        rt = self.rt
        n = proj.shape[0]
        f32 = torch.float32
        g, h, d, v = self.G, self.H, self.D, self.V
        if self.wants_f32_tokens and ctx.max_q_len == 1 and proj.dtype == f32:
            tickets = rt.workspace("delta_token_tickets", ctx.n_seqs * g, torch.int32, zero=True)
            ops.delta_token_step(proj, col0, col0 + self.b_col, col0 + self.thin_col, *self.w_second, self.conv_w, self.a_log,
                                 self.dt_bias, self.norm_w, self.eps, self.output_scale, cache.state, ctx.cu_q, ctx.slots,
                                 tickets, ctx.n_seqs, g, h, d, v, self.taps, out, y_col=out_col)
            return out
        z = self._thin_logits(proj, col0) if self.w_thin is not None else None
        decay = z if self.channel else None
        o = rt.empty(n, h * v, dtype=f32)
        if self._in_chunks(ctx) and proj.dtype == torch.bfloat16:
            need = ops.delta_chunk_buffer_bytes(n, ctx.n_seqs, h, d, v)
            buf = rt.workspace("delta_chunks", -(-need // 4), f32)                 # one buffer for all layers
            ops.delta_chunk_recurrence(proj, col0, col0 + self.b_col, self.conv_w, self.a_log, self.dt_bias, z, cache.state,
                                       ctx.cu_q, ctx.slots, ctx.n_seqs, ctx.max_q_len, g, h, d, v, self.taps, buf, o)
        else:
            qkv = rt.empty(n, self.channels, dtype=f32)
            gates = rt.empty(n, h, 2, dtype=f32)
            ops.delta_prepare(proj, self.conv_w, self.a_log, self.dt_bias, cache.state, ctx.seq_of_token, ctx.cu_q, ctx.slots,
                              ctx.n_seqs, g, h, d, v, self.taps, qkv, gates, col0=col0, b_col=col0 + self.b_col, z=decay)
            ops.delta_recurrence(qkv, gates, cache.state, ctx.cu_q, ctx.slots, ctx.n_seqs, g, h, d, v, o, z=decay)
        gate, gate_col = (z, h * d if self.channel else 0) if self.thin_gate else (proj, col0 + self.gate_col)
        if gate.dtype != f32:
            gate, gate_col = gate[:, gate_col:gate_col + h * v].to(f32).contiguous(), 0
        ops.delta_gated_norm(o, proj, self.norm_w, self.eps, g, h, d, v, out, cache.state, ctx.cu_q, ctx.slots, ctx.n_seqs,
                             self.taps, col0=col0, gate=gate, gate_col=gate_col, sigmoid=self.thin_gate,
                             scale=self.output_scale, y_col=out_col)
        return out


class LightningAttention(Part):
    """Lightning attention: linear attention with a fixed decay per head.  Per head, with a matrix state S
    [head_dim, value_dim] in FP32, zero before a request's first token:

        q = silu(W_q x), k = silu(W_k x)  (head_dim entries), v = silu(W_v x)  (value_dim entries)
        S <- decay_head * S + k v^T;   o = S^T q                           (no other scale)

    All heads' o side by side are divided by their root mean square (``norm_eps``), multiplied by a plain weight
    and by sigmoid(W_g x), and leave through W_o.  ``decay`` (one number per head) and ``value_dim`` come in the
    spec's extra.

    The four projections of x are ONE product (rows q | k | v | gate); everything from there to the gated norm is
    FP32 on the device (csrc/lightning.cu): a request's tokens of a step run in chunks whose inner products are
    written out, so a prompt portion costs matrix products instead of a chain of rank-one updates - every chunk's own
    sum at once, a scan over the chunks that leaves the state before each, every chunk's read-out at once -, and a
    step of single tokens is one launch that reads and writes every state once.  A step's kernels run exactly
    once, so the state advances by exactly the step's tokens."""

    kernel_modules = ("lightning",)       # libraries of csrc that this part's kernels live in

    adds_into_residual = True
    graph_safe = "all"

    @staticmethod
    def _dims(spec):
        e = spec.extra_dict()
        return spec.num_heads, spec.head_dim, int(e.get("value_dim", spec.head_dim))

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        h, d, v = LightningAttention._dims(spec)
        return {"q": WeightSlot((h * d, hidden_size)), "k": WeightSlot((h * d, hidden_size)),
                "v": WeightSlot((h * v, hidden_size)), "g": WeightSlot((h * v, hidden_size)),
                "o": WeightSlot((hidden_size, h * v)), "norm": WeightSlot((h * v,), init="ones")}

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        super().__init__(spec, hidden_size, weights, rt)
        h, d, v = self._dims(spec)
        decay = tuple(float(x) for x in spec.extra_dict().get("decay", ()))
        if h <= 0 or v <= 0 or len(decay) != h:
            raise ConfigError("lightning attention: heads and value size must be positive, with one decay per head")
        if not 0 < d <= ops.LIGHTNING_MAX_DIM:
            raise ConfigError(f"lightning attention: a key size of {d} is not supported (1 to {ops.LIGHTNING_MAX_DIM})")
        self.H, self.D, self.V = h, d, v
        self.eps = float(spec.extra_dict().get("norm_eps", 1e-6))
        rows = [weights[s] for s in ("q", "k", "v", "g")]
        self.gate_col = 2 * h * d + h * v
        pad = -(self.gate_col + h * v) % 8         # zero rows, so that every row of the result starts on 16 bytes
        if pad:
            rows.append(torch.zeros(pad, hidden_size, dtype=weights["q"].dtype, device=weights["q"].device))
        self.w_in = rt.weight(torch.cat(rows, dim=0))
        self.w_o = rt.weight(weights["o"])
        self.decay = torch.tensor(decay, dtype=torch.float32, device=rt.device)
        self.norm_w = rt.gain(weights["norm"])

    def cache_need(self):
        return StateNeed((self.H * self.D * self.V,), "float32")

    def weights_in_order(self) -> tuple:
        return (self.w_in, self.w_o)

    def can_fuse_norm(self, norm, n_rows: int) -> bool:
        return self.rt.skinny(n_rows, self.hidden_size) and self.rt.fuses_norm(norm)

    def forward(self, x: torch.Tensor, ctx, cache, residual=None):
        return self.finish(self.rt.linear(x, self.w_in), ctx, cache, residual=residual)

    def forward_fused_norm(self, h: torch.Tensor, norm, ctx, cache, residual=None):
        """As forward, with x = norm(h): the norm runs inside the projection (steps of a few rows)."""
        return self.finish(self.project(h, norm), ctx, cache, residual=residual)

    def project(self, h: torch.Tensor, norm) -> torch.Tensor:
        proj = self.rt.empty(h.shape[0], self.w_in.shape[0])
        ops.gemv_norm_bf16(h, norm.gain, norm.eps, None, self.w_in, proj, ops.STORE_BF16)
        return proj

    def finish(self, proj: torch.Tensor, ctx, cache, residual=None):
        rt = self.rt
        n = proj.shape[0]
        h, d, v = self.H, self.D, self.V
        o = rt.empty(n, h * v, dtype=torch.float32)
        buf = None
        if ctx.max_q_len > 1:       # chunks: every chunk's own sum, then the state before it (one buffer for all layers)
            buf = rt.workspace("lightning_chunks", ops.lightning_max_chunks(n, ctx.n_seqs) * h * d * v, torch.float32)
        ops.lightning_recurrence(proj, cache.state, ctx.cu_q, ctx.slots, ctx.n_seqs, self.decay, h, d, v, o,
                                 max_q_len=ctx.max_q_len, buf=buf)
        y = rt.empty(n, h * v)
        ops.lightning_gated_norm(o, proj, self.gate_col, self.norm_w, self.eps, y)
        return rt.linear(y, self.w_o, out_dtype=torch.float32, residual=residual)


class Retention(Part):
    """Retention: linear attention with a fixed decay per head, rotated queries and keys, no softmax and no
    denominator.  Per head, with a matrix state S [head_dim, value_dim] in FP32 that starts at zero and is carried from
    token to token for each request:

        q = rot(W_q x), k = rot(W_k x) * key_scale  (head_dim entries), v = W_v x  (value_dim entries)
        S <- decay_head * S + k v^T;   o = S^T q

    rot is the spec's position encoding (pairs (i, i + rotary_dim / 2) of the first ``rotary_dim`` dimensions of every
    head).  Each head's o is divided by its own root mean square (``norm_eps``, no weight); the heads side by side are
    multiplied by silu(W_g x) and leave through W_o.  ``decay`` (one number per head), ``value_dim`` and ``key_scale``
    (head_dim^-1/2 unless given) come in the spec's extra.

    The four projections of x are ONE product (rows q | k | v | gate).  Rotation and key scale give q, k, v in FP32
    (one kernel); from there the recurrence is the one of lightning attention without its activations
    (csrc/lightning.cu: chunk sums, scan and read-outs for prompt portions, one launch for single tokens), on the FP32
    numbers, so that rotated queries and keys are never rounded to the activations' type; the state is a slot of the
    runner's state pool."""

    kernel_modules = ("lightning",)       # libraries of csrc that this part's kernels live in

    adds_into_residual = True
    graph_safe = "all"
    # A factor on the mixer's output that whoever owns it may set (mixers side by side weight their outputs): it rides
    # in the per-head gated norm, before the output projection, which is linear.
    takes_output_scale = True
    output_scale = 1.0

    @staticmethod
    def _dims(spec):
        e = spec.extra_dict()
        return spec.num_heads, spec.head_dim, int(e.get("value_dim", spec.head_dim))

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        h, d, v = Retention._dims(spec)
        return {"q": WeightSlot((h * d, hidden_size)), "k": WeightSlot((h * d, hidden_size)),
                "v": WeightSlot((h * v, hidden_size)), "g": WeightSlot((h * v, hidden_size)),
                "o": WeightSlot((hidden_size, h * v))}

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        super().__init__(spec, hidden_size, weights, rt)
        h, d, v = self._dims(spec)
        e = spec.extra_dict()
        decay = tuple(float(x) for x in e.get("decay", ()))
        if h <= 0 or v <= 0 or len(decay) != h:
            raise ConfigError("retention: heads and value size must be positive, with one decay per head")
        if not 0 < d <= ops.LIGHTNING_MAX_DIM:
            raise ConfigError(f"retention: a key size of {d} is not supported (1 to {ops.LIGHTNING_MAX_DIM})")
        self.H, self.D, self.V = h, d, v
        self.eps = float(e.get("norm_eps", 1e-6))
        self.key_scale = float(e["key_scale"]) if e.get("key_scale") is not None else float(d) ** -0.5
        self.position = part("position", spec.position.kind)(spec.position, hidden_size, {}, rt)
        if self.position.rotary_dim > d or (self.position.rotary_dim > 0 and self.position.interleaved) or \
                getattr(self.position, "head_slopes", None) is not None or float(getattr(self.position, "magnitude", 1.0)) != 1.0:
            raise ConfigError("retention rotates the pairs (i, i + rotary_dim / 2) of at most head_dim dimensions")
        rows = [weights[s] for s in ("q", "k", "v", "g")]
        self.gate_col = 2 * h * d + h * v
        pad = -(self.gate_col + h * v) % 8         # zero rows, so that every row of the result starts on 16 bytes
        if pad:
            rows.append(torch.zeros(pad, hidden_size, dtype=weights["q"].dtype, device=weights["q"].device))
        self.w_in = rt.weight(torch.cat(rows, dim=0))
        self.w_o = rt.weight(weights["o"])
        self.decay = torch.tensor(decay, dtype=torch.float32, device=rt.device)

    def cache_need(self):
        return StateNeed((self.H * self.D * self.V,), "float32")

    def weights_in_order(self) -> tuple:
        return (self.w_in, self.w_o)

    def forward(self, x: torch.Tensor, ctx, cache, residual=None):
        return self.finish(self.rt.linear(x, self.w_in), ctx, cache, residual=residual)

    def finish(self, proj: torch.Tensor, ctx, cache, residual=None):
        rt = self.rt
        n = proj.shape[0]
        h, d, v = self.H, self.D, self.V
        f32 = torch.float32
        o = rt.empty(n, h * v, dtype=f32)
        if ctx.max_q_len == 1:      # single tokens: rotation, key scale, state update and read-out in one launch
            ops.retention_token_step(proj, cache.state, ctx.cu_q, ctx.slots, ctx.n_seqs, self.decay, h, d, v, o,
                                     ctx.positions, self.position.inv_freq, self.position.rotary_dim, self.key_scale)
        else:
            qkv = rt.empty(n, self.gate_col, dtype=f32)
            ops.linear_attention_prepare(proj, ctx.positions, self.position.inv_freq, self.key_scale, qkv, h, d, v,
                                         self.position.rotary_dim)
            # chunks: every chunk's own sum, then the state before it (one buffer for all layers)
            buf = rt.workspace("lightning_chunks", ops.lightning_max_chunks(n, ctx.n_seqs) * h * d * v, f32)
            ops.lightning_recurrence(qkv, cache.state, ctx.cu_q, ctx.slots, ctx.n_seqs, self.decay, h, d, v, o,
                                     max_q_len=ctx.max_q_len, buf=buf, activation=False)
        y = rt.empty(n, h * v)
        ops.group_gated_norm(o, proj, self.gate_col, None, self.eps, y, v, gate="silu", scale=self.output_scale)
        return rt.linear(y, self.w_o, out_dtype=f32, residual=residual)


class MatrixMemory(Part):
    """A matrix memory with exponential gates (the mLSTM cell of xLSTM).  Per head, with a matrix S [head_dim, value_dim], a
    normaliser n [head_dim] and a running maximum m, all FP32 and zero at a sequence's start:

        q = W_q x * head_dim^-1/2, k = W_k x, v = W_v x
        i = cap tanh((W_i x + b_i) / cap),  f = logsigmoid(cap tanh((W_f x + b_f) / cap))       (one number per head each)
        m' = max(f + m, i);   S <- e^(f + m - m') S + e^(i - m') k v^T;   n <- e^(f + m - m') n + e^(i - m') k;   m <- m'
        o = S^T q / (max(|n . q|, e^-m) + 1e-6)

    Each head's o is divided by its own root mean square (``norm_eps``), multiplied by a weight over all heads ("norm") and
    by sigmoid(W_g x), and leaves through W_o.  ``value_dim`` and ``gate_cap`` come in the spec's extra.

    A step of single tokens is one FP32-out product for everything the layer projects and ONE launch for the rest
    (csrc/mlstm.cu).  Other steps run in chunks: the queries, keys, values and output gates in the compute type, the
    logits of i and f as a product of their own that leaves in FP32; every chunk's own sum, a scan, every chunk's
    read-out.  The state is a slot of the runner's state pool."""

    kernel_modules = ("mlstm", "lightning")       # libraries of csrc that this part's kernels live in

    adds_into_residual = True
    graph_safe = "all"

    @staticmethod
    def _dims(spec):
        e = spec.extra_dict()
        return spec.num_heads, spec.head_dim, int(e.get("value_dim", spec.head_dim))

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        h, d, v = MatrixMemory._dims(spec)
        return {"q": WeightSlot((h * d, hidden_size)), "k": WeightSlot((h * d, hidden_size)),
                "v": WeightSlot((h * v, hidden_size)), "g": WeightSlot((h * v, hidden_size)),
                "o": WeightSlot((hidden_size, h * v)), "norm": WeightSlot((h * v,), init="ones"),
                "i": WeightSlot((h, hidden_size)), "i.b": WeightSlot((h,)),
                "f": WeightSlot((h, hidden_size)), "f.b": WeightSlot((h,))}

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        super().__init__(spec, hidden_size, weights, rt)
        h, d, v = self._dims(spec)
        e = spec.extra_dict()
        if h <= 0 or v <= 0:
            raise ConfigError("matrix memory: heads and value size must be positive")
        if not 0 < d <= ops.MLSTM_MAX_DIM:
            raise ConfigError(f"matrix memory: a key size of {d} is not supported (1 to {ops.MLSTM_MAX_DIM})")
        self.H, self.D, self.V = h, d, v
        self.eps, self.cap = float(e.get("norm_eps", 1e-6)), float(e["gate_cap"])
        if not self.cap > 0.0:
            raise ConfigError("matrix memory: gate_cap must be positive")
        self.q_scale = float(d) ** -0.5

        def padded(names):
            rows = [weights[s] for s in names]
            pad = -sum(r.shape[0] for r in rows) % 8         # zero rows, so that every row of the result starts on 16 bytes
            if pad:
                rows.append(torch.zeros(pad, hidden_size, dtype=weights["q"].dtype, device=weights["q"].device))
            return rows

        wide, narrow = padded(("q", "k", "v", "g")), padded(("i", "f"))
        self.n_wide = sum(r.shape[0] for r in wide)
        self.w_in = rt.weight(torch.cat(wide + narrow, dim=0))          # q | k | v | gate | pad | i | f | pad
        self.w_o = rt.weight(weights["o"])
        self.norm_w = rt.gain(weights["norm"])
        self.bias_i, self.bias_f = rt.gain(weights["i.b"]), rt.gain(weights["f.b"])

    def cache_need(self):
        return StateNeed((ops.mlstm_state_floats(self.H, self.D, self.V),), "float32")

    def weights_in_order(self) -> tuple:
        return (self.w_in, self.w_o)

    def forward(self, x: torch.Tensor, ctx, cache, residual=None):
        rt = self.rt
        n = x.shape[0]
        h, d, v = self.H, self.D, self.V
        f32 = torch.float32
        y = rt.empty(n, h * v)
        gates = (self.bias_i, self.bias_f, self.cap, cache.state, ctx.cu_q, ctx.slots, ctx.n_seqs)
        if ctx.max_q_len == 1:
            proj = rt.linear(x, self.w_in, out_dtype=f32)
            ops.mlstm_token_step(proj, proj, self.n_wide, self.n_wide + h, *gates, self.q_scale, self.norm_w, self.eps, y, h, d, v)
        else:
            proj = rt.linear(x, self.w_in[:self.n_wide])
            z = rt.linear(x, self.w_in[self.n_wide:], out_dtype=f32)
            buf = rt.workspace("mlstm_chunks", ops.mlstm_buffer_floats(n, ctx.n_seqs, h, d, v), f32)     # one for all layers
            out = rt.empty(n, h * v, dtype=f32)
            ops.mlstm_chunk_step(proj, z, 0, h, *gates, ctx.max_q_len, self.q_scale, self.norm_w, self.eps, buf, out, y, h, d, v)
        return rt.linear(y, self.w_o, out_dtype=f32, residual=residual)


register_part("mixer", "matrix_memory", MatrixMemory, replace=True)
register_part("mixer", "gated_delta", GatedDeltaRule, replace=True)
register_part("mixer", "retention", Retention, replace=True)
register_part("mixer", "lightning", LightningAttention, replace=True)
