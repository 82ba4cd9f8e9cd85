"""A decoder-only model as data plus parts: embedding, a list of blocks, the
order in which they run, a final norm and an output head.

Nothing here is specific to an architecture; an architecture only supplies the
ModelSpec.  The part order of one step is the reference's
(crates/forward/README.md:18-39): embed, the layer calls, then final norm and
head on the wanted rows only (crates/forward/src/core/composites/output_head.rs:32-57).
"""
from __future__ import annotations

import torch

from ..cache.manager import CallPlan
from ..parts.block import ResidualStream
from ..parts.spec import ModelSpec, build_part


class DecoderModel:
    def __init__(self, spec: ModelSpec, runtime):
        spec.validate()
        self.spec = spec
        self.runtime = runtime
        self.hidden_size, self.vocab_size = spec.hidden_size, spec.vocab_size
        self.embedding = build_part(spec.embedding, runtime)
        self.layers = [build_part(s, runtime) for s in spec.layers]
        self.order = list(spec.order)
        self.final_norm = build_part(spec.final_norm, runtime)
        self.head = build_part(spec.head, runtime)
        self.reentry = build_part(spec.reentry, runtime) if spec.reentry is not None else None

    # ---- weights -----------------------------------------------------------
    def parts(self):
        return [p for p in (self.embedding, self.reentry, *self.layers, self.final_norm, self.head) if p is not None]

    def tensor_specs(self) -> dict:
        specs = {}
        for p in self.parts():
            for name, ts in p.tensor_specs().items():
                if name in specs and specs[name].shape != ts.shape:
                    raise ValueError(f"two parts want tensor '{name}' with different shapes")
                specs[name] = ts
        return specs

    def shared_tensor_names(self) -> set:
        """Tensors that more than one part wants (a table of which every layer reads its own columns): they are kept on
        the device once."""
        seen, shared = set(), set()
        for p in self.parts():
            names = set(p.tensor_specs())
            shared |= seen & names
            seen |= names
        return shared

    def bind(self, tensors: dict) -> None:
        for p in self.parts():
            p.bind(tensors)

    def graph_safe(self) -> bool:
        return all(p.all_graph_safe() for p in self.parts())

    def step_weight_bytes(self) -> int:
        """Bytes of weights one step reads: every layer call's weights once, the final norm and the head."""
        total = self.final_norm.weight_bytes() + self.head.weight_bytes()
        for call in self.order:
            total += self.layers[call.layer].weight_bytes()
            if call.reenter:
                total += self.reentry.weight_bytes()
        return total

    # ---- what the cache manager must provide ---------------------------------
    def cache_plans(self) -> list:
        plans = []
        for call in self.order:
            block = self.layers[call.layer]
            mixer = block.mixer
            # (a block that keeps state beside its mixer's, such as the inputs a convolution still needs, says so)
            state = block.state_requirement() if hasattr(block, "state_requirement") else mixer.state_requirement()
            plans.append(CallPlan(kv=mixer.cache_requirement(), state=state, cache_from=call.cache_from))
        # an embedding that keeps something per request (the token before, say) has an entry behind the layer calls
        state = self._embedding_state()
        if state is not None:
            plans.append(CallPlan(state=state))
        return plans

    def _embedding_state(self):
        return self.embedding.state_requirement() if hasattr(self.embedding, "state_requirement") else None

    # ---- one step -------------------------------------------------------------
    def forward(self, ctx) -> torch.Tensor | None:
        """Runs the rows of ctx.batch; returns float32 logits [n_out, vocab] (None when nothing is wanted)."""
        rt, b = self.runtime, ctx.batch
        n = b.n_tokens
        x = ctx.open_stream(self.hidden_size)
        if self._embedding_state() is not None:
            self.embedding.forward(ctx, b.token_ids[:n], x, state=ctx.cache(len(self.order)).state)
        else:
            self.embedding.forward(ctx, b.token_ids[:n], x)
        stream = ResidualStream(x)
        x0 = None
        if self.reentry is not None:
            # the embedding output is wanted again later: the layers work on a copy of it (one device-to-device copy)
            x0 = x
            stream.x = ctx.step_alloc((n, self.hidden_size), torch.float32)
            stream.x.copy_(x0)
        for ci, call in enumerate(self.order):
            if call.reenter:
                self.reentry.forward(ctx, stream, x0, call.pass_index)
            self.layers[call.layer].forward(ctx, stream, ci)
        if b.n_out == 0:
            return None
        stream.close(ctx)         # (a block arrangement that kept the stream as several copies folds them into one)
        h = ctx.step_alloc((b.n_out, self.hidden_size), rt.dtype)
        self.final_norm.add_norm(ctx, stream.x, stream.pending, h, rows=b.out_rows[:b.n_out],
                                 n_partials=stream.pending_slabs, delta_norm=stream.pending_norm)
        logits = ctx.logits(b.n_out, self.vocab_size)
        self.head.forward(ctx, h, logits)
        return logits
