"""Linear attention with data-dependent decays: the gated delta rule, and gated linear attention.

Every head keeps a float32 state ``S`` [head_dim, value_dim] a request, zero at position 0.

``gated_delta``: ``q, k, v`` (q and k with ``num_qk_heads`` heads, head h reads q/k head ``h // (num_heads / num_qk_heads)``)
each pass a causal convolution a channel (``conv_kernel`` taps, the last on the current token, no bias) and silu; q
and k become unit vectors a head (1e-6 joins the sum of squares under the root), q times ``head_dim^-1/2``; ``beta = sigmoid(h Wb^T)``, one
a head; then every row decays the state, corrects what it holds for the row's key, and reads the corrected state:

    F = g S_before ;  e = beta (v - F^T k) ;  S = F + k e^T ;  o = S^T q .

``decay`` = ``"head"``: one factor a head, ``g = exp(-exp(A_log) softplus(h Wa^T + dt_bias))``; ``"channel"``: one a key
channel (a row of S), with the low-rank projection ``(h Wa1^T) Wa2^T`` in the place of ``h Wa^T`` and ``dt_bias``
[num_heads * head_dim].  Every head's o is divided by its root mean square, times a weight [value_dim] shared by the heads,
times ``gate``: ``"silu"`` (``silu(h Wg^T)``) or ``"sigmoid"``, the projection whole (``gate_rank`` = "full") or low-rank
(``"low"``: ``(h Wg1^T) Wg2^T``); then the output matrix.  Ranks are taken from the tensors' shapes.

``gated_linear``: ``q = h Wq^T head_dim^-1/2``, ``k``, ``v`` with as many heads each and no convolution; a factor a key
channel ``g = sigmoid(z)^(1/tau)``, ``z = (h Wa1^T) Wa2^T + b``; each row multiplies the state's rows by their factors, adds ``k v^T`` and reads with q;
the same norm a head, times ``silu(h Wg^T)``, then the output matrix.

Everything that reads the layer's input is one product; what enters the recurrence behind the projections (unit norms,
step sizes, decays) and the recurrence itself are float32 (csrc/recurrence.cu).  Decoded tokens and short portions run the
scan kernel (row after row, the same bits however a sequence is cut; the 32-bit mode runs it always); in 16-bit mode a
step with a portion of ``CHUNKED_FROM`` rows or more runs the chunked kernels, whose list of chunks is the step table
that the ``lightning`` mixer builds too.  A request keeps the states of the heads and, with convolutions, their last
``conv_kernel - 1`` inputs, as one float32 row in its slot.

``out_scale`` (default 1) multiplies the mixer's output (carried by the norm's weight): for mixers that are summed.

Params of ``gated_delta``: hidden_size, num_heads, num_qk_heads, head_dim, value_dim, conv_kernel, norm_eps, decay, gate,
gate_rank, out_scale; of ``gated_linear``: hidden_size, num_heads, head_dim, value_dim, tau, norm_eps, out_scale.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..cache.spec import StateSpec
from ..config.schema import ConfigError
from ..ops import kernels as K
from ..ops.linear import linear
from .base import Part, WeightSpec, register_part
from .lightning import lightning_chunks


class RowLayout:
    """Row stretches of one wide matrix, each starting on a multiple of 8 rows (a stretch of the product's output then
    starts on a 16-byte boundary and can be a matrix operand itself)."""

    def __init__(self):
        self.rows, self.col, self.n = [], {}, 0

    def add(self, name: str, w: torch.Tensor, multiple: int = 8) -> None:
        self.col[name] = self.n
        pad = -w.shape[0] % multiple
        self.rows.append(w)
        if pad:
            self.rows.append(torch.zeros((pad, w.shape[1]), dtype=w.dtype, device=w.device))
        self.n += w.shape[0] + pad

    def matrix(self) -> torch.Tensor:
        return torch.cat(self.rows, 0).contiguous()


LOW_RANK_MULTIPLE = 32      # a low-rank product's inner size is padded with zeros up to a multiple of this (what its kernels take)


def pad_columns(w: torch.Tensor, multiple: int = LOW_RANK_MULTIPLE) -> torch.Tensor:
    pad = -w.shape[1] % multiple
    if not pad:
        return w.contiguous()
    return torch.cat([w, torch.zeros((w.shape[0], pad), dtype=w.dtype, device=w.device)], 1).contiguous()


class _Recurrence(Part):
    """What the two mixers share: the choice between scan and chunks, the norm and gate behind them."""

    category = "mixer"
    graph_safe = True

    def _sizes(self, what: str) -> None:
        self.d = int(self._p("hidden_size"))
        self.H = int(self._p("num_heads"))
        self.G = int(self._p("num_qk_heads", self.H))
        self.D = int(self._p("head_dim"))
        self.P = int(self._p("value_dim", self.D))
        self.eps = float(self._p("norm_eps"))
        self.out_scale = float(self._p("out_scale", 1.0))
        if min(self.H, self.G, self.D, self.P) < 1:
            raise ConfigError(f"{what}: heads and sizes must be positive")
        if self.H % self.G:
            raise ConfigError(f"{what}: num_heads={self.H} must be a multiple of num_qk_heads={self.G}")
        if self.D > K.RECUR_MAX_DIM:
            raise ConfigError(f"{what}: head_dim={self.D} is not supported by the kernels (at most {K.RECUR_MAX_DIM})")
        self.state_len = self.H * self.D * self.P
        self.chunked = self.env.dtype != torch.float32 and K.recur_chunks_ok(self.D, self.P) and self.env.device.type == "cuda"
        if self.chunked:
            self.chunk_rows = K.recur_chunk_rows()
            self.step_tables_key = ("lightning_chunks", self.chunk_rows)

    def step_tables(self, segs):
        return lightning_chunks(segs, self.chunk_rows)

    def _bind_out(self, w):
        self.w_o = w["out_proj.weight"].contiguous()
        self.norm_w = (w["norm.weight"].float() * self.out_scale).repeat(self.H).contiguous()

    def _recur(self, q, k, v, lg, beta, q_scale, per_channel, ctx, cache):
        """The recurrence over the step's rows; float32 [n, num_heads * value_dim]."""
        sizes = (self.H, self.G, self.D, self.P, per_channel, cache.writes)
        o = torch.empty((ctx.n_rows, self.H * self.P), dtype=torch.float32, device=q.device)
        chunks = ctx.tables.get(self.step_tables_key) if self.chunked else None
        scan = lambda n_seg: K.recur_scan(q, k, v, lg, beta, q_scale, cache.tensor, ctx.cu_rows, ctx.seg_pos, ctx.seg_slot, o, n_seg, *sizes)
        if chunks is not None:
            nl = chunks.n_lead
            if nl:
                scan(nl)                                         # decoded tokens beside the portions: the scan takes them
            K.recur_chunks(q, k, v, lg, beta, q_scale, cache.tensor, ctx.cu_rows[nl:], ctx.seg_pos[nl:], ctx.seg_slot[nl:],
                           chunks.chunk_seg, chunks.chunk_row0, chunks.seg_chunk0, chunks.n_chunks, o, ctx.n_seg - nl, *sizes)
        else:
            scan(ctx.n_seg)
        return o

    def _finish(self, o, gate, act, residual):
        og = torch.empty(o.shape, dtype=gate.dtype, device=o.device)
        K.group_norm_gate_rows(o, self.norm_w, gate, self.eps, og, self.H, False, act)
        linear(og, self.w_o, out=residual, accumulate=True)

    # (a mixer whose first product can be run together with others': see parallel.py)
    def input_product(self):
        return self.w_in, None

    def drop_input_product(self):
        self.w_in = None

    def forward(self, h, residual, ctx, cache):
        """``cache``: a :class:`~kappai_b200.cache.storage.StateView`; a slot's row begins with the heads' states."""
        self.forward_projected(linear(h, self.w_in), residual, ctx, cache)


class GatedDelta(_Recurrence):
    def __init__(self, params, env):
        super().__init__(params, env)
        self._sizes("gated_delta")
        self.taps = int(self._p("conv_kernel"))
        self.decay = self._p("decay", "head")
        self.gate = self._p("gate", "silu")
        self.gate_rank = self._p("gate_rank", "full")
        for name, value, known in (("decay", self.decay, ("head", "channel")), ("gate", self.gate, ("silu", "sigmoid")),
                                   ("gate_rank", self.gate_rank, ("full", "low"))):
            if value not in known:
                raise ConfigError(f"gated_delta: {name}='{value}' (expected '{known[0]}' or '{known[1]}')")
        if not (1 <= self.taps <= K.RECUR_MAX_TAPS):
            raise ConfigError(f"gated_delta: conv_kernel={self.taps} outside 1..{K.RECUR_MAX_TAPS}")
        self.per_channel = self.decay == "channel"
        self.C = 2 * self.G * self.D + self.H * self.P            # channels of the convolution

    def weight_specs(self) -> Dict[str, WeightSpec]:
        d, H, GD, HP = self.d, self.H, self.G * self.D, self.H * self.P
        n_dec = H * self.D if self.per_channel else H
        s = {}
        for n, rows in (("q", GD), ("k", GD), ("v", HP)):
            s[f"{n}_proj.weight"] = WeightSpec((rows, d))
            s[f"{n}_conv.weight"] = WeightSpec((rows, self.taps), "conv")
        s.update({"beta_proj.weight": WeightSpec((H, d)), "A_log": WeightSpec((H,), "bias"), "dt_bias": WeightSpec((n_dec,), "bias"),
                  "norm.weight": WeightSpec((self.P,), "norm"), "out_proj.weight": WeightSpec((d, HP))})
        if self.per_channel:
            s["decay_down.weight"] = WeightSpec((-1, d), free=self.D)
            s["decay_up.weight"] = WeightSpec((H * self.D, -1), free=self.D)
        else:
            s["decay_proj.weight"] = WeightSpec((H, d))
        if self.gate_rank == "low":
            s["gate_down.weight"] = WeightSpec((-1, d), free=self.P)
            s["gate_up.weight"] = WeightSpec((HP, -1), free=self.P)
        else:
            s["gate_proj.weight"] = WeightSpec((HP, d))
        return s

    def bind(self, w):
        lay = RowLayout()
        lay.add("conv", torch.cat([w[f"{n}_proj.weight"] for n in ("q", "k", "v")], 0))
        if self.gate_rank == "full":
            lay.add("gate", w["gate_proj.weight"])
        small = [w["beta_proj.weight"]] + ([] if self.per_channel else [w["decay_proj.weight"]])
        lay.add("beta", torch.cat(small, 0))
        self.w_decay = self.w_gate = None
        if self.per_channel:
            _check_rank("gated_delta", w["decay_down.weight"], w["decay_up.weight"])
            lay.add("decay", w["decay_down.weight"], LOW_RANK_MULTIPLE)
            self.w_decay = pad_columns(w["decay_up.weight"])
        if self.gate_rank == "low":
            _check_rank("gated_delta", w["gate_down.weight"], w["gate_up.weight"])
            lay.add("gate", w["gate_down.weight"], LOW_RANK_MULTIPLE)
            self.w_gate = pad_columns(w["gate_up.weight"])
        self.w_in, self.col = lay.matrix(), lay.col
        self.conv_w = torch.cat([w[f"{n}_conv.weight"].float() for n in ("q", "k", "v")], 0).contiguous()
        self.neg_a = (-torch.exp(w["A_log"].double())).float().contiguous()
        self.dt_bias = w["dt_bias"].float().contiguous()
        self._bind_out(w)

    def cache_spec(self):
        return StateSpec((self.state_len + (self.taps - 1) * self.C,), "float32")

    def forward_projected(self, p, residual, ctx, cache):
        """``p``: the rows of the input product (``input_product``), possibly columns of a wider one."""
        H, G, D, P, n = self.H, self.G, self.D, self.P, ctx.n_rows
        f32 = dict(dtype=torch.float32, device=p.device)
        qkv = torch.empty((n, self.C), **f32)
        beta = torch.empty((n, H), **f32)
        if self.per_channel:
            a0 = self.col["decay"]
            lg = linear(p[:, a0:a0 + self.w_decay.shape[1]], self.w_decay, out_dtype=torch.float32)
        else:
            lg = torch.empty((n, H), **f32)
        b0 = self.col["beta"]
        K.delta_prep(p, self.col["conv"], b0, b0 + H, self.conv_w, self.neg_a, self.dt_bias, cache.tensor[:, self.state_len:], ctx.row_seg,
                     ctx.cu_rows, ctx.seg_pos, ctx.seg_slot, qkv, beta, lg, ctx.n_seg, H, G, D, P, float(D) ** -0.5, self.per_channel,
                     ctx.decode_only, cache.writes)
        o = self._recur(qkv[:, :G * D], qkv[:, G * D:2 * G * D], qkv[:, 2 * G * D:], lg, beta, 1.0, self.per_channel, ctx, cache)
        g0 = self.col["gate"]
        gate = p[:, g0:g0 + H * P] if self.w_gate is None else linear(p[:, g0:g0 + self.w_gate.shape[1]], self.w_gate)
        self._finish(o, gate, self.gate, residual)


class GatedLinear(_Recurrence):
    def __init__(self, params, env):
        super().__init__(params, env)
        self._sizes("gated_linear")
        self.tau = float(self._p("tau"))
        if self.G != self.H:
            raise ConfigError("gated_linear: queries and keys have as many heads as the values")
        if not self.tau > 0:
            raise ConfigError(f"gated_linear: tau={self.tau} must be positive")

    def weight_specs(self) -> Dict[str, WeightSpec]:
        d, HD, HP = self.d, self.H * self.D, self.H * self.P
        return {"q_proj.weight": WeightSpec((HD, d)), "k_proj.weight": WeightSpec((HD, d)), "v_proj.weight": WeightSpec((HP, d)),
                "gate_proj.weight": WeightSpec((HP, d)), "decay_down.weight": WeightSpec((-1, d), free=16),
                "decay_up.weight": WeightSpec((HD, -1), free=16), "decay_up.bias": WeightSpec((HD,), "bias"),
                "norm.weight": WeightSpec((self.P,), "norm"), "out_proj.weight": WeightSpec((d, HP))}

    def bind(self, w):
        lay = RowLayout()
        for n in ("q", "k", "v", "gate"):
            lay.add(n, w[f"{n}_proj.weight"])
        _check_rank("gated_linear", w["decay_down.weight"], w["decay_up.weight"])
        lay.add("decay", w["decay_down.weight"], LOW_RANK_MULTIPLE)
        self.w_in, self.col = lay.matrix(), lay.col
        self.w_decay = pad_columns(w["decay_up.weight"])
        self.b_decay = w["decay_up.bias"].float().contiguous()
        self._bind_out(w)

    def cache_spec(self):
        return StateSpec((self.state_len,), "float32")

    def forward_projected(self, p, residual, ctx, cache):
        col, HD, HP = self.col, self.H * self.D, self.H * self.P
        lg = linear(p[:, col["decay"]:col["decay"] + self.w_decay.shape[1]], self.w_decay, self.b_decay, out_dtype=torch.float32)
        K.log_decay_sigmoid(lg, self.tau)
        o = self._recur(p[:, col["q"]:col["q"] + HD], p[:, col["k"]:col["k"] + HD], p[:, col["v"]:col["v"] + HP], lg, None,
                        float(self.D) ** -0.5, True, ctx, cache)
        self._finish(o, p[:, col["gate"]:col["gate"] + HP], "silu", residual)


def _check_rank(what: str, down: torch.Tensor, up: torch.Tensor) -> None:
    if down.shape[0] != up.shape[1]:
        raise ConfigError(f"{what}: a low-rank projection goes down to {down.shape[0]} and up from {up.shape[1]}")


register_part("mixer", "gated_delta", GatedDelta)
register_part("mixer", "gated_linear", GatedLinear)
