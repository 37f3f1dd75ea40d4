"""A decoder put together from a :class:`~ginfer_b200.parts.plan.ModelPlan`.

The reference's forward pass (``ginfer/model/model.cc:152-166,180-228``): embedding, the layers
in order, final norm over all rows, row selection, LM head.  Here the layers run in the order of
the plan's run list, each run with the cache binding the plan names for it, and the final norm
is computed only at the rows whose logits are wanted.
"""
from __future__ import annotations

import torch

from .base import MixedInput, StepContext, Summed, TensorSpec, make_part
from .plan import ModelPlan


class DecoderModel:
    def __init__(self, plan: ModelPlan):
        plan.validate()
        self.plan = plan
        self.embedding = make_part("embedding", plan.embedding)
        self.blocks = [make_part("block", ls.block, layer_spec=ls) for ls in plan.layers]
        self.final_norm = make_part("norm", plan.final_norm)
        self.head = make_part("head", plan.head)
        self.stream_inputs = [make_part("stream_input", s) for s in plan.stream_inputs]
        self.dtype: torch.dtype | None = None
        self.device: torch.device | None = None

    # ------------------------------------------------------------------ tensors
    def tensor_specs(self) -> list[TensorSpec]:
        """Every tensor of the model under its full name."""
        out = list(self.embedding.tensor_specs())
        shared: dict[str, TensorSpec] = {}

        def whole_model(s: TensorSpec) -> None:
            # a tensor of the whole model ("/name"): several parts may name it, alike
            g = TensorSpec(s.name[1:], s.shape, s.role, s.int_high)
            if shared.setdefault(g.name, g) != g:
                raise ValueError(f"parts disagree about the tensor {g.name!r}: {shared[g.name]} "
                                 f"and {g}")
        for ls, blk in zip(self.plan.layers, self.blocks):
            pre = ls.prefix + "." if ls.prefix else ""
            for s in blk.tensor_specs():
                if s.name.startswith("/"):
                    whole_model(s)
                else:
                    out.append(TensorSpec(pre + s.name, s.shape, s.role, s.int_high))
        for part in self.stream_inputs:
            for s in part.tensor_specs():
                if s.name.startswith("/"):
                    whole_model(s)
                else:
                    out.append(s)
        out += list(shared.values())
        out += self.final_norm.tensor_specs()
        out += self.head.tensor_specs()
        names = [s.name for s in out]
        if len(set(names)) != len(names):
            dup = sorted({n for n in names if names.count(n) > 1})
            raise ValueError(f"the plan names these tensors more than once: {dup}")
        return out

    def load(self, tensors: dict[str, torch.Tensor], dtype: torch.dtype,
             device: torch.device) -> None:
        self.dtype, self.device = dtype, device
        self.embedding.load(tensors, dtype, device)
        whole = {"/" + k: v for k, v in tensors.items()}       # tensors of the whole model
        for ls, blk in zip(self.plan.layers, self.blocks):
            pre = ls.prefix + "." if ls.prefix else ""
            local = {k[len(pre):]: v for k, v in tensors.items() if k.startswith(pre)}
            local.update(whole)
            blk.load(local, dtype, device)
        for part in self.stream_inputs:
            part.load({**tensors, **whole}, dtype, device)
        self.final_norm.load(tensors, dtype, device)
        self.head.load(tensors, dtype, device)

    # ------------------------------------------------------------------ caches
    def cache_specs(self) -> dict[int, object]:
        """Cache id -> spec, taken from the layer whose run writes that cache."""
        def of_mixer(e) -> tuple:
            spec = self.blocks[e.layer].mixer.cache_spec()
            specs = spec if isinstance(spec, tuple) else (spec,)
            if len(specs) != len(e.caches()):
                raise ValueError(f"a run of layer {e.layer} names {len(e.caches())} caches; its mixer "
                                 f"keeps {len(specs)}")
            return specs
        out: dict[int, object] = {}
        own = self.embedding.state_spec()
        if (own is None) != (self.plan.embedding_state is None):
            raise ValueError("the plan and the embedding disagree on whether it keeps a state")
        if own is not None:
            out[self.plan.embedding_state] = own
        for e in self.plan.run:
            if e.write_cache:
                out.update(zip(e.caches(), of_mixer(e)))
            own = self.blocks[e.layer].state_spec()
            if (own is None) != (e.block_state is None):
                raise ValueError(f"a run of layer {e.layer} and its block disagree on whether the "
                                 "block keeps a state")
            if own is not None:
                out[e.block_state] = own
        for e in self.plan.run:
            if not e.write_cache:
                for c, mine in zip(e.caches(), of_mixer(e)):
                    if mine != out[c]:
                        raise ValueError(f"layer {e.layer} cannot read cache {c}: it holds "
                                         f"{out[c]} but the layer expects {mine}")
        return out

    def _next_input(self, blk, entry, own_state):
        """What ``blk`` may prepare for ``entry``'s run behind it: nothing where that run's block needs
        its own state for it and the state is not at hand, or where ``blk`` does not know how."""
        if entry.block_state is not None and own_state is None:
            return None
        first = self.blocks[entry.layer].first_input(own_state)
        if isinstance(first, MixedInput) and not blk.prepares_mixed_input:
            return None
        return first

    # ------------------------------------------------------------------ one step
    def forward(self, ctx: StepContext, bind_cache) -> torch.Tensor:
        """Run the step's tokens; ``bind_cache(run_entry)`` gives the cache binding of a run,
        ``bind_cache(run_entry, block=True)`` that of its block's own state, ``bind_cache(id)`` that
        of a state by its number.
        Returns fp32 logits ``[R, vocab]`` at ``ctx.logit_rows``."""
        delta = None
        own = {}
        if self.plan.embedding_state is not None:
            own["own_state"] = bind_cache(self.plan.embedding_state)
        x = self.embedding.forward(ctx.token_ids, ctx, **own)
        embedded = x
        run = self.plan.run
        for i, e in enumerate(run):
            blk = self.blocks[e.layer]
            if e.enter is not None:
                if delta is not None:
                    x, delta = x.float() + delta.float(), None
                x = self.stream_inputs[e.enter[0]].enter(x, ctx, embedded, e.enter[1])
            kw = {}
            if e.block_state is not None:
                kw["own_state"] = bind_cache(e, block=True)
            if blk.takes_next_norm and i + 1 < len(run) and run[i + 1].enter is None:
                # the block may prepare the input of the norm that the next run starts with
                n = run[i + 1]
                own = None
                if n.block_state is not None and blk.prepares_shifted_input:
                    own = bind_cache(n, block=True)
                x, delta = blk.forward(x, delta, ctx, bind_cache(e),
                                       then=self._next_input(blk, n, own), **kw)
            else:
                x, delta = blk.forward(x, delta, ctx, bind_cache(e), **kw)
        if ctx.logit_rows.numel() == 0:
            return torch.empty((0, self.plan.vocab_size), dtype=torch.float32, device=ctx.device)
        if isinstance(x, Summed):
            _, n = self.final_norm.forward(x.tensor, None, rows=ctx.logit_rows, want_sum=False,
                                           out_dtype=ctx.dtype)
        else:
            _, n = self.final_norm.forward(x, delta, rows=ctx.logit_rows, want_sum=False,
                                           out_dtype=ctx.dtype)
        return self.head.forward(n, ctx)
