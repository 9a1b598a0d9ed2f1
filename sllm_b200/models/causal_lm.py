"""The generic causal language model: embedding, a run list of blocks built from
a `ModelPlan`, a final norm and an output head.  It knows no architecture; the
plan decides which parts stand where and in which order they run.
"""

from __future__ import annotations

import torch

from .. import ops
from ..config.plan import ModelPlan
from ..parts import delta_rule as _delta_rule, experts as _experts, latent_attention as _latent  # noqa: F401
from ..parts import linear_attention as _linear_attention, parallel as _parallel, side_by_side as _side_by_side  # noqa: F401
from ..parts import gated_recurrence as _gated_recurrence, output_norm as _output_norm, sandwich as _sandwich  # noqa: F401
from ..parts import hyper_connections as _hyper_connections, state_space as _state_space  # noqa: F401
from ..parts import standard as _standard  # noqa: F401  (each import registers its parts)
from ..parts.base import (BLOCKS, COMPLETE, FEED_FORWARDS, MIXERS, NORMS, POSITIONS, SHIFTS,
                          LayerCache, SlotState, StepContext, TensorSpec, flatten_needs, join_name)


PREVIOUS_TOKEN = "previous_token"        # the model's own per-request state (see `CausalLM.cache_needs`)
FAMILIES = {"mixer": MIXERS, "feed_forward": FEED_FORWARDS, "norm": NORMS, "shift": SHIFTS}


class Layer:
    """The parts a `LayerSpec` names, built, and the block that arranges them.  The block receives
    them by role and says what the layer wants of the cache manager."""

    def __init__(self, spec, *, dtype, device):
        self.spec = spec
        self.parts = {role: FAMILIES[e.family].build(e.spec, dtype=dtype, device=device) for role, e in spec.parts.items()}
        self.block = BLOCKS.get(spec.block)(self.parts)

    @property
    def mixer(self):
        return self.parts.get("mixer")

    def cache_need(self):
        return self.block.cache_need()

    def named_parts(self):
        s = self.spec
        return [(join_name(s.prefix, e.name), self.parts[role]) for role, e in s.parts.items()]


class CausalLM:
    def __init__(self, plan: ModelPlan, *, dtype: torch.dtype, device):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"compute dtype must be bfloat16 or float32, got {dtype}")
        plan.validate()
        self.plan = plan
        self.dtype = dtype
        self.device = torch.device(device)
        kw = dict(dtype=dtype, device=self.device)
        self.layers = [Layer(s, **kw) for s in plan.layers]
        self.final_norm = NORMS.build(plan.final_norm, **kw)
        self.embedding_norm = NORMS.build(plan.embedding_norm, **kw) if plan.embedding_norm is not None else None
        self.pass_vectors = None   # [passes, H] float32
        self.token_table = None    # [V, width] compute dtype: vectors that belong to a token
        self.pair_table = None     # [buckets + 1, H] compute dtype: rows by pairs of tokens
        self.stream_sum = torch.ones(plan.streams, dtype=torch.float32, device=self.device) if plan.streams is not None else None
        self.position = POSITIONS.build(plan.position, **kw) if plan.position is not None else None
        self.embedding = None      # [V, H] compute dtype
        self.head = None           # [V, H] compute dtype (the embedding itself when tied)

    # ---- weights ---------------------------------------------------------------
    def _named_parts(self):
        out = []
        for layer in self.layers:
            out.extend(layer.named_parts())
        out.append((self.plan.final_norm_name, self.final_norm))
        if self.embedding_norm is not None:
            out.append((self.plan.embedding_norm_name, self.embedding_norm))
        if self.position is not None and self.plan.position_name:
            out.append((self.plan.position_name, self.position))
        return out

    def tensor_specs(self) -> list[TensorSpec]:
        p = self.plan
        specs = [TensorSpec(p.embedding_name, (p.vocab_size, p.hidden_size), role="embedding")]
        for prefix, part in self._named_parts():
            specs.extend(s.prefixed(prefix) for s in part.tensor_specs())
        if p.head_name is not None:
            specs.append(TensorSpec(p.head_name, (p.vocab_size, p.hidden_size), role="matrix"))
        if p.pass_vectors_name is not None:
            specs.append(TensorSpec(p.pass_vectors_name, (p.passes, p.hidden_size), role="bias"))
        if p.token_table_name is not None:
            specs.append(TensorSpec(p.token_table_name, (p.vocab_size, p.token_table_width), role="embedding"))
        if p.token_pairs is not None:
            specs.append(TensorSpec(p.token_pairs.name, (p.token_pairs.buckets + 1, p.hidden_size), role="embedding"))
        return specs

    def ignored_tensor_names(self):
        """Tensors a checkpoint may carry that this model does not use (the plan names them)."""
        return list(self.plan.ignored_names)

    def bind(self, fetch) -> None:
        p = self.plan
        self.embedding = fetch(p.embedding_name).to(device=self.device, dtype=self.dtype).contiguous()
        for prefix, part in self._named_parts():
            part.bind(lambda rel, _p=prefix: fetch(join_name(_p, rel)))
        if p.pass_vectors_name is not None:
            self.pass_vectors = fetch(p.pass_vectors_name).to(device=self.device, dtype=torch.float32).contiguous()
        if p.token_table_name is not None:
            self.token_table = fetch(p.token_table_name).to(device=self.device, dtype=self.dtype).contiguous()
            for _, part in self._named_parts():
                if hasattr(part, "adopt_token_table"):
                    part.adopt_token_table(self.token_table)
        if p.token_pairs is not None:
            self.pair_table = fetch(p.token_pairs.name).to(device=self.device, dtype=self.dtype).contiguous()
        if p.head_name is None:
            self.head = self.embedding
        else:
            self.head = fetch(p.head_name).to(device=self.device, dtype=self.dtype).contiguous()

    def weight_bytes(self) -> int:
        """Bytes of every tensor a decode step reads once (the head counts once
        more when it is the embedding table: the step reads it whole as the head
        and only single rows of it as the embedding)."""
        n = self.head.numel() * self.head.element_size()
        runs = {}
        for e in self.plan.run_list:            # a layer that runs several times in a step is read as often
            runs[e.layer] = runs.get(e.layer, 0) + 1
        for i, layer in enumerate(self.layers):
            n += runs.get(i, 0) * sum(part.weight_bytes() for _, part in layer.named_parts())
        n += self.final_norm.weight_bytes()
        if self.embedding_norm is not None:
            n += self.embedding_norm.weight_bytes()
        if self.position is not None and self.plan.position_name:
            n += self.position.weight_bytes()
        return n

    # ---- cache needs ----------------------------------------------------------------
    def cache_needs(self):
        """One entry per run of the run list: the mixer's need, or the index of
        the run whose cache it borrows.  What the model itself keeps per request (the token before, where the
        embedding takes in pairs) rides with the first run."""
        out = []
        for e in self.plan.run_list:
            if e.cache_from is not None:
                # the pages are borrowed; what the layer keeps per request beside them (a convolution's last inputs) is its own
                own = tuple(n for n in flatten_needs(self.layers[e.layer].cache_need()) if isinstance(n, SlotState))
                out.append(("borrow", e.cache_from, own) if own else ("borrow", e.cache_from))
            else:
                out.append(("own", self.layers[e.layer].cache_need()))
        if self.plan.token_pairs is not None:
            out[0] = ("own", tuple(flatten_needs(out[0][1])) + (SlotState((1,), PREVIOUS_TOKEN),))
        return out

    # ---- forward ------------------------------------------------------------------
    def forward(self, step: StepContext, caches: list[LayerCache]) -> torch.Tensor:
        """Run the batch's tokens through every entry of the run list and return
        float32 logits ``[R, V]`` at ``step.logit_rows``."""
        p = self.plan
        if p.token_pairs is None and p.streams is None:
            residual = ops.embed_gather(self.embedding, step.token_ids, p.embedding_scale)           # [T, H] float32
        else:
            before = caches[0].states[PREVIOUS_TOKEN] if p.token_pairs is not None else None
            residual = ops.embed_streams(self.embedding, step, p.embedding_scale, p.streams, self.pair_table, before, p.token_pairs)
        if self.position is not None:
            self.position.on_embedding(residual, step)
        entered = None
        if self.embedding_norm is not None:
            # the normed rows are the stream's start; a range of layers that runs again takes them in once more
            entered = self.embedding_norm.add_norm(residual, None, out_dtype=torch.float32)
            residual = entered.clone() if any(e.reentry for e in self.plan.run_list) else entered
        delta = None
        runs = self.plan.run_list
        for i, e in enumerate(runs):
            block = self.layers[e.layer].block
            if e.reentry is not None:
                # (a term the run before left pending is added by this block's norm; sums commute)
                ops.add_rows_(residual, entered if e.reentry > 0 else None, self.pass_vectors[e.reentry])
            kw = {}
            if getattr(block, "accepts_next_norm", False) and i + 1 < len(runs):
                # the norm that reads the stream next: this block's last product may prepare its input
                kw["next_norm"] = getattr(self.layers[runs[i + 1].layer].block, "first_norm", None)
            delta = block.forward(residual, delta, step, caches[i], self.position, write_cache=e.cache_from is None, **kw)
        if p.streams is not None:
            if step.logit_rows.numel() == 0:
                return torch.empty((0, p.vocab_size), dtype=torch.float32, device=self.device)
            x = _hyper_connections.read_streams(residual, delta, step.logit_rows, self.stream_sum, self.final_norm, self.dtype)
            return self._logits(x)
        if isinstance(delta, COMPLETE):          # (a block handed one on although nothing asked: take the stream as it is)
            delta = None
        if step.logit_rows.numel() == 0:
            return torch.empty((0, self.plan.vocab_size), dtype=torch.float32, device=self.device)
        res_rows = ops.gather_rows(residual, step.logit_rows)
        delta_rows = ops.gather_rows(delta, step.logit_rows) if delta is not None else None
        x = self.final_norm.add_norm(res_rows, delta_rows)
        return self._logits(x)

    def _logits(self, x: torch.Tensor) -> torch.Tensor:
        logits = ops.linear(x, self.head, None, torch.float32)
        return ops.softcap_(logits, self.plan.logit_softcap) if self.plan.logit_softcap is not None else logits
