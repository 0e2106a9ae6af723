"""Arrangements of a mixer, a feed-forward and their norms around the residual.

``prenorm_residual``: ``x += mixer(norm1(x)); x += ffn(norm2(x))``
(src/models/lfm.c:7-53 followed by src/recipe/builders.c:378-388).  The
residual ``x`` is float32 and is updated in place.  A ``side`` part, if the
layer has one, then changes the residual once more (``side.forward(x, ctx)``).

``postnorm_residual``: ``x <- norm1(alpha x + mixer(x)); x <- norm2(alpha x + ffn(x))``:
the sublayers read ``x`` itself (in the compute type), the norm comes after the
sum, and ``alpha`` (parameter, default 1) weighs the residual branch.  A layer
without a feed-forward has the first half only.  The sum and the norm are
float32; one kernel norms a sum and writes what the next sublayer needs (its
input in the compute type and ``alpha`` times the new residual to add into), so
a layer costs two row-wise launches, as a pre-norm layer does.

``parallel_residual``: ``h = norm1(x); x += mixer(h); x += ffn(h)``: one norm a
layer, and both sublayers read its output.  Each sublayer adds its float32
output into the float32 residual, so the layer's sum is
``(x + mixer(h)) + ffn(h)``.

``sandwich_residual``: ``x += norm1b(mixer(norm1(x))); x += norm2b(ffn(norm2(x)))``:
a norm in front of every sublayer and one behind it, before its output joins the
residual.  The sublayer adds its float32 output into a zeroed float32 branch;
one kernel norms the branch, adds it to the residual, clears the branch for
its next use and, where another norm follows at once (the feed-forward's, or
the first norm of the layer that runs next), norms the new residual for it in
the same pass.

``gated_residual``: ``h = norm1(x); x += ls1 * sigmoid(h Wg1^T + b1) * mixer(h)``, the
same with norm2, ls2, Wg2, b2 for the feed-forward: a sublayer's output is scaled
a channel (``layer_scale``; tensors ``ls1``, ``ls2`` [hidden]) and gated element by
element by its own input (``gate``; ``rg1.weight`` [hidden, hidden] and ``rg1.bias``,
and so on), either of which may be off.  The sublayer adds into a zeroed
float32 branch; one kernel scales and gates it into the residual, clears it and
norms the residual for the sublayer that follows (of this layer or the one that
runs next).  Where the mixer offers its first product, the gate's rows run in it.

``streams_residual``: the residual is several float32 streams a row (streams.py).
A sublayer reads ``norm(sum_b in_b x_b)`` and its output y joins every stream
while the streams are mixed, ``x'_b = out_b y + sum_a mix_ab x_a``; mixer
and feed-forward each with coefficients of their own (``hc1``, ``hc2``:
``in`` [streams], ``out`` [streams], ``mix`` [streams, streams], indexed from,
to).  As above a sublayer adds into a zeroed float32 branch, and one kernel
reads the branch, changes the streams, clears the branch and norms the weighted
sum that the next sublayer reads (of this layer or the one that runs next).
"""
from __future__ import annotations

import torch

from ..config.schema import ConfigError
from ..ops import kernels as K
from ..ops.linear import linear
from .base import Part, WeightSpec, register_part
from .streams import stream_norm


class PreNormResidualBlock(Part):
    category = "block"
    graph_safe = True

    def assemble(self, mixer, ffn, mixer_norm, ffn_norm, side=None):
        self.mixer, self.ffn, self.mixer_norm, self.ffn_norm, self.side = mixer, ffn, mixer_norm, ffn_norm, side
        return self

    def forward(self, x, ctx, cache):
        self.mixer.forward(self.mixer_norm.forward(x) if self.mixer_norm is not None else x, x, ctx, cache)
        if self.ffn is not None:
            self.ffn.forward(self.ffn_norm.forward(x) if self.ffn_norm is not None else x, x, ctx)
        if self.side is not None:
            self.side.forward(x, ctx)


class PostNormResidualBlock(Part):
    category = "block"
    graph_safe = True

    def __init__(self, params, env):
        super().__init__(params, env)
        self.alpha = float(self._p("alpha", 1.0))

    def assemble(self, mixer, ffn, mixer_norm, ffn_norm, side=None):
        if mixer_norm is None or (ffn is not None and ffn_norm is None):
            raise ValueError("postnorm_residual: every sublayer needs the norm that follows its sum")
        if side is not None:
            raise ValueError("postnorm_residual: no side part in this arrangement")
        self.mixer, self.ffn, self.mixer_norm, self.ffn_norm, self.side = mixer, ffn, mixer_norm, ffn_norm, None
        return self

    def _enter(self, x, ctx):
        """The sublayer input (x in the compute type) and alpha * x: left by the block before this one for
        this very residual, or made here."""
        carry = getattr(ctx, "postnorm_carry", None)
        ctx.postnorm_carry = None
        if carry is not None and carry[0] is x and carry[1] == self.alpha:
            return carry[2], carry[3]
        acc = torch.empty_like(x)
        if self.env.dtype == torch.float32:
            K.scale_cast(x, None, acc, self.alpha)
            return x, acc
        h = torch.empty(x.shape, dtype=self.env.dtype, device=x.device)
        K.scale_cast(x, h, acc, self.alpha)
        return h, acc

    def forward(self, x, ctx, cache):
        f32 = self.env.dtype == torch.float32
        h, acc = self._enter(x, ctx)
        self.mixer.forward(h, acc, ctx, cache)
        # what the sublayer after this norm reads and adds into; in 32-bit its input is the residual itself
        h2 = x if f32 else (h if h is not x else torch.empty(x.shape, dtype=self.env.dtype, device=x.device))
        if self.ffn is not None:
            n1 = self.mixer_norm
            K.postnorm_rows(acc, n1.weight, n1.eps, x_out=x if f32 else None, h_out=None if f32 else h2,
                            scaled_out=acc, alpha=self.alpha)
            self.ffn.forward(h2, acc, ctx)
            last = self.ffn_norm
        else:
            last = self.mixer_norm
        # the new residual, and with it the entry of a post-norm block that may follow
        K.postnorm_rows(acc, last.weight, last.eps, x_out=x, h_out=None if f32 else h2, scaled_out=acc, alpha=self.alpha)
        ctx.postnorm_carry = (x, self.alpha, x if f32 else h2, acc)


class ParallelResidualBlock(Part):
    category = "block"
    graph_safe = True

    def assemble(self, mixer, ffn, mixer_norm, ffn_norm, side=None):
        if ffn_norm is not None:
            raise ValueError("parallel_residual: the sublayers share one norm")
        self.mixer, self.ffn, self.mixer_norm, self.ffn_norm, self.side = mixer, ffn, mixer_norm, None, side
        return self

    def forward(self, x, ctx, cache):
        if self.mixer_norm is not None:
            h = self.mixer_norm.forward(x)
        elif self.env.dtype == torch.float32:
            h = x.clone()                      # the sublayers add into x while the second still has to read its input
        else:
            h = K.cast(x, torch.empty(x.shape, dtype=self.env.dtype, device=x.device))
        self.mixer.forward(h, x, ctx, cache)
        if self.ffn is not None:
            self.ffn.forward(h, x, ctx)
        if self.side is not None:
            self.side.forward(x, ctx)


def branch_rows(n, d, ctx, device):
    """The float32 rows a sublayer adds its output into: one zeroed buffer a step, shared by the layers (the
    kernel that reads a branch clears it)."""
    y = getattr(ctx, "branch_buffer", None)
    if y is None or tuple(y.shape) != (n, d):
        y = torch.zeros((n, d), dtype=torch.float32, device=device)
        ctx.branch_buffer = y
    return y


class SandwichResidualBlock(Part):
    category = "block"
    graph_safe = True

    def assemble(self, mixer, ffn, mixer_norm, ffn_norm, side=None, post_norms=(None, None)):
        p1, p2 = post_norms
        if mixer_norm is None or p1 is None or (ffn is not None and (ffn_norm is None or p2 is None)):
            raise ValueError("sandwich_residual: every sublayer needs a norm in front and a norm behind")
        if any(type(n).__name__ != "RMSNorm" for n in (mixer_norm, p1, ffn_norm, p2) if n is not None):
            raise ValueError("sandwich_residual: the norms are RMS norms")
        self.mixer, self.ffn, self.mixer_norm, self.ffn_norm, self.side = mixer, ffn, mixer_norm, ffn_norm, side
        self.mixer_post_norm, self.ffn_post_norm = p1, p2
        return self

    def forward(self, x, ctx, cache):
        y = branch_rows(x.shape[0], x.shape[1], ctx, x.device)
        # the input of this layer's mixer: left by the layer before for this very residual, or made here
        carry = getattr(ctx, "sandwich_carry", None)
        ctx.sandwich_carry = None
        n1 = self.mixer_norm
        if carry is not None and carry[0] is x and carry[1] is n1:
            h = carry[2]
        else:
            h = n1.forward(x)
        self.mixer.forward(h, y, ctx, cache)
        if self.ffn is not None:
            n2, pn = self.ffn_norm, self.mixer_post_norm
            h2 = torch.empty(x.shape, dtype=self.env.dtype, device=x.device)
            K.rmsnorm_add_norm_rows(y, pn.weight, pn.eps, x, n2.weight, n2.eps, h2)
            self.ffn.forward(h2, y, ctx)
            last = self.ffn_post_norm
        else:
            last = self.mixer_post_norm
        nxt = getattr(ctx, "next_block", None)
        if isinstance(nxt, SandwichResidualBlock) and self.side is None:
            nn = nxt.mixer_norm
            h_next = torch.empty(x.shape, dtype=self.env.dtype, device=x.device)
            K.rmsnorm_add_norm_rows(y, last.weight, last.eps, x, nn.weight, nn.eps, h_next)
            ctx.sandwich_carry = (x, nn, h_next)
        else:
            K.rmsnorm_add_norm_rows(y, last.weight, last.eps, x)
        if self.side is not None:
            self.side.forward(x, ctx)


class StreamsResidualBlock(Part):
    category = "block"
    graph_safe = True

    def __init__(self, params, env):
        super().__init__(params, env)
        self.S = int(self._p("streams"))
        self.sublayers = int(self._p("sublayers", 2))           # 1: a layer without a feed-forward

    def weight_specs(self):
        S = self.S
        return {f"hc{q}.{n}": WeightSpec(shape, "stream") for q in range(1, self.sublayers + 1)
                for n, shape in (("in", (S,)), ("out", (S,)), ("mix", (S, S)))}

    def bind(self, w):
        self.hc = [{n: w[f"hc{q}.{n}"].float().contiguous() for n in ("in", "out", "mix")} for q in range(1, self.sublayers + 1)]

    def assemble(self, mixer, ffn, mixer_norm, ffn_norm, side=None):
        if side is not None:
            raise ValueError("streams_residual: no side part in this arrangement")
        if self.sublayers != (1 if ffn is None else 2):
            raise ValueError("streams_residual: coefficients for every sublayer the layer has, and no more")
        self.mixer, self.ffn, self.mixer_norm, self.ffn_norm, self.side = mixer, ffn, mixer_norm, ffn_norm, None
        self.centred = [stream_norm(n) for n in (mixer_norm, ffn_norm)[:self.sublayers]]
        return self

    def _step(self, x, y, q, nxt, j, last):
        """Sublayer q's output y joins the streams; the normed input of block ``nxt``'s sublayer j leaves (unless ``last``)."""
        hc = self.hc[q]
        if last:
            K.streams_rows(x, y, hc["mix"], hc["out"])
            return None
        norm = (nxt.mixer_norm, nxt.ffn_norm)[j]
        h = torch.empty((x.shape[0], x.shape[2]), dtype=self.env.dtype, device=x.device)
        K.streams_rows(x, y, hc["mix"], hc["out"], nxt.hc[j]["in"], norm.weight, norm.eps, nxt.centred[j], h)
        return h

    def forward(self, x, ctx, cache):
        """``x``: float32 [rows, streams, hidden]."""
        y = branch_rows(x.shape[0], x.shape[2], ctx, x.device)
        carry = getattr(ctx, "streams_carry", None)
        ctx.streams_carry = None
        if carry is not None and carry[0] is x and carry[1] is self:
            h = carry[2]
        else:
            h = torch.empty((x.shape[0], x.shape[2]), dtype=self.env.dtype, device=x.device)
            n1 = self.mixer_norm
            K.streams_rows(x, in_w=self.hc[0]["in"], norm_w=n1.weight, eps=n1.eps, centred=self.centred[0], h=h)
        self.mixer.forward(h, y, ctx, cache)
        q = 0
        if self.ffn is not None:
            h = self._step(x, y, 0, self, 1, False)
            self.ffn.forward(h, y, ctx)
            q = 1
        nxt = getattr(ctx, "next_block", None)
        follows = isinstance(nxt, StreamsResidualBlock) and nxt.S == self.S
        h = self._step(x, y, q, nxt, 0, not follows)
        if follows:
            ctx.streams_carry = (x, nxt, h)


class GatedResidualBlock(Part):
    category = "block"
    graph_safe = True

    def __init__(self, params, env):
        super().__init__(params, env)
        self.d = int(self._p("hidden_size"))
        self.sublayers = int(self._p("sublayers", 2))           # 1: a layer without a feed-forward
        self.layer_scale = bool(self._p("layer_scale", True))
        self.gate = bool(self._p("gate", True))

    def weight_specs(self):
        s = {}
        for q in range(1, self.sublayers + 1):
            if self.layer_scale:
                s[f"ls{q}"] = WeightSpec((self.d,), "norm")
            if self.gate:
                s[f"rg{q}.weight"] = WeightSpec((self.d, self.d))
                s[f"rg{q}.bias"] = WeightSpec((self.d,), "bias")
        return s

    def assemble(self, mixer, ffn, mixer_norm, ffn_norm, side=None):
        if side is not None:
            raise ConfigError("gated_residual: no side part in this arrangement")
        if self.sublayers != (1 if ffn is None else 2):
            raise ConfigError("gated_residual: tensors for every sublayer the layer has, and no more")
        if any(type(n).__name__ != "RMSNorm" for n in (mixer_norm, ffn_norm)[:self.sublayers]):
            raise ConfigError("gated_residual: every sublayer has an RMS norm in front")
        self.mixer, self.ffn, self.mixer_norm, self.ffn_norm, self.side = mixer, ffn, mixer_norm, ffn_norm, None
        return self

    def bind(self, w):
        # (the mixer's own weights are bound already: a layer's parts are bound in the order in which they are made)
        n = self.sublayers
        self.ls = [w[f"ls{q}"].float().contiguous() if self.layer_scale else None for q in range(1, n + 1)]
        self.w_g = [w[f"rg{q}.weight"].contiguous() if self.gate else None for q in range(1, n + 1)]
        self.b_g = [w[f"rg{q}.bias"].float().contiguous() if self.gate else None for q in range(1, n + 1)]
        self.w_in = self.b_in = None
        offered = self.mixer.input_product() if self.gate and hasattr(self.mixer, "input_product") else None
        if offered is not None and offered[0].dtype == self.w_g[0].dtype:
            w_m, b_m = offered
            self.cols = w_m.shape[0]
            b_m = b_m if b_m is not None else torch.zeros(self.cols, dtype=torch.float32, device=w_m.device)
            # (zero rows behind the last, so that a row of the product's output starts on a 16-byte boundary)
            pad = -(self.cols + self.d) % 8
            self.w_in = torch.cat([w_m, self.w_g[0], w_m.new_zeros((pad, self.d))], 0).contiguous()
            self.b_in = torch.cat([b_m, self.b_g[0], b_m.new_zeros(pad)]).contiguous()
            self.mixer.drop_input_product()
            self.w_g[0] = self.b_g[0] = None

    def _close(self, x, y, gate, q, norm):
        """Sublayer q's output y joins the residual; with ``norm`` the normed residual leaves."""
        if norm is None:
            K.gated_add_norm_rows(y, gate, self.ls[q], x)
            return None
        h = torch.empty(x.shape, dtype=self.env.dtype, device=x.device)
        K.gated_add_norm_rows(y, gate, self.ls[q], x, norm.weight, norm.eps, h)
        return h

    def forward(self, x, ctx, cache):
        y = branch_rows(x.shape[0], x.shape[1], ctx, x.device)
        # the input of this layer's mixer: left by the layer before for this very residual, or made here
        carry = getattr(ctx, "gated_carry", None)
        ctx.gated_carry = None
        h = carry[2] if carry is not None and carry[0] is x and carry[1] is self.mixer_norm else self.mixer_norm.forward(x)
        gate = None
        if self.w_in is not None:
            p = linear(h, self.w_in, self.b_in)
            gate = p[:, self.cols:self.cols + self.d]
            self.mixer.forward_projected(p[:, :self.cols], y, ctx, cache)
        else:
            if self.gate:
                gate = linear(h, self.w_g[0], self.b_g[0])
            self.mixer.forward(h, y, ctx, cache)
        q = 0
        if self.ffn is not None:
            h = self._close(x, y, gate, 0, self.ffn_norm)
            gate = linear(h, self.w_g[1], self.b_g[1]) if self.gate else None
            self.ffn.forward(h, y, ctx)
            q = 1
        nxt = getattr(ctx, "next_block", None)
        follows = isinstance(nxt, GatedResidualBlock)
        h = self._close(x, y, gate, q, nxt.mixer_norm if follows else None)
        if follows:
            ctx.gated_carry = (x, nxt.mixer_norm, h)


register_part("block", "gated_residual", GatedResidualBlock)
register_part("block", "streams_residual", StreamsResidualBlock)
register_part("block", "sandwich_residual", SandwichResidualBlock)
register_part("block", "prenorm_residual", PreNormResidualBlock)
register_part("block", "parallel_residual", ParallelResidualBlock)
register_part("block", "postnorm_residual", PostNormResidualBlock)
