"""The gated delta rule: a recurrent mixer with a matrix of state per head."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Mixer, StateRequirement, TensorSpec
from .linear import Linear, concat_rows
from .spec import register_part


class GatedDeltaRule(Mixer):
    """A linear recurrence over a request's tokens.  With H value heads on G query/key heads (head h reads q/k head
    h // (H / G)), key size dk and value size dv:

        q = Wq x, k = Wk x  [G][dk];   v = Wv x  [H][dv]                          (no biases)
        each channel of q, k and v passes a causal convolution over the last `conv` tokens (its own taps, the last
        tap is the current token's, zeros before the request's start) and then SiLU
        q <- q / sqrt(sum q^2 + unit_eps) * dk^-1/2,  k <- k / sqrt(sum k^2 + unit_eps)        (per head)
        beta = sigmoid(Wb x)  [H];     g = exp(-exp(A_log) * softplus(Wa x + dt_bias))  [H]
        per head, token by token:  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
        o <- o / sqrt(mean(o^2) + eps) * norm * silu(Wg x)_head                    (norm [dv] shared by the heads)
        out = Wo [o_0 ; ... ; o_{H-1}]

    `decay` 'channel': one decay per head and key channel, S <- diag(g) S with
        g = exp(-exp(A_log)_head * softplus(Wa2 (Wa1 x) + dt_bias))  [H][dk]          (through a narrow middle)
    `gate` 'sigmoid': sigmoid takes the place of silu on the gate; `low_rank_gate`: the gate's map is Wg2 (Wg1 x).  The
    widths of the middles are the sizes of the tensors (no configuration key gives them; `rank` is what the
    random-weights mode draws).

    S [dk, dv] starts at zero and is carried from step to step in float32, as are the last conv - 1 inputs of the
    convolution: both live in the request's state slot (one float32 array: S for every head, then the tail).  Decays,
    beta, the unit norms, the recurrence and the head norm are float32 in both engine modes.

    The input maps are one stacked product (q, k, v, the narrow middles, beta, a, gate); the maps behind the middles are
    one kernel with their functions.  Tensors behind the prefix: q, q.conv, k, k.conv, v, v.conv ([channels, conv]), b
    ([H, width]), A_log ([H]), dt_bias ([H], or [H * dk] with a decay per channel), a ([H, width]) or a1 ([Ra, width]) and
    a2 ([H * dk, Ra]), g ([H * dv, width]) or g1 ([Rg, width]) and g2 ([H * dv, Rg]), norm ([dv]), o."""
    graph_safe = True

    def __init__(self, runtime=None, prefix="", *, width: int, num_heads: int, num_qk_heads: int, key_dim: int,
                 value_dim: int, conv: int = 4, eps: float = 1e-6, unit_eps: float = 1e-6, init_std: float = 0.02,
                 decay: str = "head", gate: str = "silu", low_rank_gate: bool = False, rank: int = 16):
        super().__init__(runtime, prefix)
        self.width, self.H, self.G = int(width), int(num_heads), int(num_qk_heads)
        self.dk, self.dv, self.taps = int(key_dim), int(value_dim), int(conv)
        if self.H % self.G:
            raise ValueError(f"{self.H} value heads are not a multiple of {self.G} query/key heads")
        if self.taps < 1:
            raise ValueError("the short convolution needs at least one tap")
        self.eps, self.unit_eps, self.init_std = float(eps), float(unit_eps), init_std
        if decay not in ("head", "channel") or gate not in ("silu", "sigmoid"):
            raise ValueError(f"gated delta rule: decay {decay!r} ('head', 'channel'), gate {gate!r} ('silu', 'sigmoid')")
        self.by_channel, self.gate, self.low_rank_gate, self.rank = decay == "channel", gate, bool(low_rank_gate), int(rank)
        self.qk, self.vw = self.G * self.dk, self.H * self.dv
        self.channels = 2 * self.qk + self.vw                    # what passes the convolution
        self.state_floats = self.H * self.dk * self.dv
        self.tail_floats = (self.taps - 1) * self.channels
        self.slot_floats = -(-(self.state_floats + self.tail_floats) // 4) * 4         # (slots start on 16-byte borders)
        self.proj = self.o = self.conv_w = self.a_log = self.dt_bias = self.norm = self.a2 = self.g2 = None

    def state_requirement(self):
        return StateRequirement((self.slot_floats,), "float32")

    def own_tensor_specs(self):
        p, init = self.prefix, ("normal", self.init_std)
        conv_init = ("normal", 0.5 / max(1, self.taps) ** 0.5)
        specs = {
            p + "q": TensorSpec((self.qk, self.width), init=init),
            p + "q.conv": TensorSpec((self.qk, self.taps), init=conv_init),
            p + "k": TensorSpec((self.qk, self.width), init=init),
            p + "k.conv": TensorSpec((self.qk, self.taps), init=conv_init),
            p + "v": TensorSpec((self.vw, self.width), init=init),
            p + "v.conv": TensorSpec((self.vw, self.taps), init=conv_init),
            p + "b": TensorSpec((self.H, self.width), init=init),
            p + "A_log": TensorSpec((self.H,), init=("normal", 0.5)),
            p + "dt_bias": TensorSpec((self.H * (self.dk if self.by_channel else 1),), init=("normal", 0.5)),
            p + "norm": TensorSpec((self.dv,), init=("one_plus_normal", 0.1)),
            p + "o": TensorSpec((self.width, self.vw), init=init),
        }
        if self.by_channel:
            specs[p + "a1"] = TensorSpec((self.rank, self.width), init=init, free_axes=(0,))
            specs[p + "a2"] = TensorSpec((self.H * self.dk, self.rank), init=("normal", 0.5), free_axes=(1,))
        else:
            specs[p + "a"] = TensorSpec((self.H, self.width), init=init)
        if self.low_rank_gate:
            specs[p + "g1"] = TensorSpec((self.rank, self.width), init=init, free_axes=(0,))
            specs[p + "g2"] = TensorSpec((self.vw, self.rank), init=("normal", 0.5), free_axes=(1,))
        else:
            specs[p + "g"] = TensorSpec((self.vw, self.width), init=init)
        return specs

    def own_bind(self, tensors):
        p = self.prefix
        # the narrow middles right behind q, k and v: their columns then start on 16-byte borders where the sizes allow it
        names = ["q", "k", "v"] + (["a1"] if self.by_channel else []) + (["g1"] if self.low_rank_gate else []) + ["b"] \
            + ([] if self.by_channel else ["a"]) + ([] if self.low_rank_gate else ["g"])
        stack = [tensors[p + n] for n in names]
        self.offset, rows = {}, 0
        for name, t in zip(names, stack):
            self.offset[name] = rows
            rows += t.shape[0]
        for first, second in (("a1", "a2"), ("g1", "g2")):
            if first in names and tensors[p + first].shape[0] != tensors[p + second].shape[1]:
                raise ValueError(f"{p}{first} has {tensors[p + first].shape[0]} outputs, {p}{second} takes "
                                 f"{tensors[p + second].shape[1]} inputs")
        if rows % 8:          # rows of zeros up to a multiple of 8, so that the product's float32 rows stay 16-byte aligned
            stack.append(torch.zeros((8 - rows % 8, self.width), dtype=stack[0].dtype, device=stack[0].device))
        self.proj = Linear(concat_rows(stack))
        self.o = Linear(tensors[p + "o"])
        self.conv_w = torch.cat([tensors[p + "q.conv"], tensors[p + "k.conv"], tensors[p + "v.conv"]]).contiguous()
        if self.by_channel:
            self.a2 = tensors[p + "a2"].contiguous()
        if self.low_rank_gate:
            self.g2 = tensors[p + "g2"].contiguous()
            if self.by_channel and self.g2.dtype != self.a2.dtype:
                self.g2 = self.g2.to(self.a2.dtype)
        dt = self.a2.dtype if self.by_channel else self.conv_w.dtype
        self.a_log, self.dt_bias = tensors[p + "A_log"].to(dt).contiguous(), tensors[p + "dt_bias"].to(dt).contiguous()
        self.norm = tensors[p + "norm"]

    def own_weights(self):
        return [self.proj.weight, self.o.weight, self.conv_w] + [t for t in (self.a2, self.g2) if t is not None]

    def forward(self, ctx, h, out, call):
        n = ctx.n_tokens
        rt, b = self.runtime, ctx.batch
        state = ctx.cache(call).state
        if state is None:
            raise ValueError("the gated delta rule needs a state slot per request")
        state = state.view(state.shape[0], -1)
        off = self.offset
        with ctx.ws.scope():
            slabs = ctx.ws.alloc((ctx.max_slabs, n, self.proj.out_features), torch.float32)
            parts = self.proj.slabs(ctx, h, slabs)
            stride = slabs.stride(0)
            qkv = ctx.ws.alloc((n, self.channels), torch.float32)
            beta = ctx.ws.alloc((n, self.H), torch.float32)
            decay = ctx.ws.alloc((n, self.H * (self.dk if self.by_channel else 1)), torch.float32)
            per_head = not self.by_channel
            ops.gdr_prepare(slabs[0], self.conv_w, self.taps, self.a_log if per_head else None,
                            self.dt_bias if per_head else None, state, self.state_floats, b, qkv, beta,
                            decay if per_head else None, self.G, self.H, self.dk, self.dv, self.dk ** -0.5, self.unit_eps,
                            n_partials=parts, partial_stride=stride, b_off=off["b"], a_off=off.get("a"))
            maps, gate = [], None
            if self.by_channel:
                maps.append(ops.LowRankMap(self.a2, off["a1"], decay, "decay", bias=self.dt_bias, log_rate=self.a_log,
                                           group=self.dk))
            if self.low_rank_gate:
                gate = ctx.ws.alloc((n, self.vw), torch.float32)
                maps.append(ops.LowRankMap(self.g2, off["g1"], gate))
            if maps:
                ops.low_rank_maps(slabs[0], maps, n_partials=parts, partial_stride=stride)
            o = ctx.ws.alloc((n, self.vw), torch.float32)
            recurrent = ops.gdr_channel_recurrent if self.by_channel else ops.gdr_recurrent
            recurrent(qkv, beta, decay, state, b, o, self.G, self.H, self.dk, self.dv)
            a = ctx.ws.alloc((n, self.vw), rt.dtype)
            if gate is not None:
                ops.gdr_out_norm(o, gate, 0, self.norm, self.eps, a, self.H, self.dv, gate=self.gate)
            else:
                ops.gdr_out_norm(o, slabs[0], off["g"], self.norm, self.eps, a, self.H, self.dv, n_partials=parts,
                                 partial_stride=stride, gate=self.gate)
            ctx.to_stream(self.o, a)


register_part("mixer", "gated_delta", GatedDeltaRule)
