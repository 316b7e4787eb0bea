"""A causal language model assembled from a ``ModelPlan``.

Owns the parts and the map from checkpoint tensor names to the parts' local
names.  ``forward`` runs the plan's schedule over the tokens of one step and
returns float32 logits at the wanted rows (final norm and head run on those rows
only; the reference norms every row first, src/inference.cu:68-69).
"""
from __future__ import annotations

from typing import Callable, Mapping

import torch

from ..config.plan import ModelPlan
from .base import FixedStateSpec, PagedKVSpec, Part, WeightSpec, build_part


class CausalLM:
    def __init__(self, plan: ModelPlan):
        self.plan = plan
        self.embedding = build_part("embedding", plan.embedding)
        self.final_norm = build_part("norm", plan.final_norm)
        self.head = build_part("head", plan.head)
        self.blocks = []
        self._named: list[tuple[str, Part]] = [
            (plan.names["embedding"], self.embedding),
            (plan.names["final_norm"], self.final_norm),
            (plan.names["head"], self.head),
        ]
        self.junction = None
        if plan.junction is not None:
            self.junction = build_part("junction", plan.junction)
            self._named.append((plan.names["junction"], self.junction))
        for lp in plan.layers:
            parts = {
                "mixer": build_part("mixer", lp.mixer),
                "ffn": None if lp.ffn is None else build_part("ffn", lp.ffn),
                "mixer_norm": build_part("norm", lp.mixer_norm),
                "ffn_norm": None if lp.ffn_norm is None else build_part("norm", lp.ffn_norm),
            }
            for role, spec in (("mixer_post_norm", lp.mixer_post_norm), ("ffn_post_norm", lp.ffn_post_norm)):
                if spec is not None:             # only blocks that norm a sublayer's output take these
                    parts[role] = build_part("norm", spec)
            self.blocks.append(build_part("block", lp.block, **parts))
            if "block" in lp.names:            # an arrangement with tensors of its own
                self._named.append((lp.names["block"], self.blocks[-1]))
            for role, part in parts.items():
                if part is not None:
                    self._named.append((lp.names[role], part))

    # ---- weights -------------------------------------------------------------------------
    def expected_tensors(self) -> dict[str, WeightSpec]:
        """Checkpoint name -> shape and initialisation class of every tensor the model needs."""
        out: dict[str, WeightSpec] = {}
        for prefix, part in self._named:
            for local, spec in part.weight_specs().items():
                out[prefix + local] = spec
        return out

    def duplicate_tensors(self) -> dict[str, str]:
        """Checkpoint names the model does not need but a folder may still hold, each with the
        name of the tensor it repeats: a tied head's own table beside the embedding's (some
        published checkpoints with tied embeddings store the table twice).  The reference never
        reads a head of its own (src/model.cpp:120-121)."""
        if getattr(self.head, "tied", False):
            local = getattr(self.embedding, "tensor", "weight")
            return {self.plan.names["head"] + "weight": self.plan.names["embedding"] + local}
        return {}

    def load_weights(self, fetch: Callable[[str], torch.Tensor], ops, present=None) -> None:
        """``fetch(name)`` returns the checkpoint tensor on the device, dtype as stored;
        ``present(name)`` (if given) says whether the source holds a tensor: an optional one
        that it lacks reaches its part as None."""
        for prefix, part in self._named:
            names = part.weight_specs()
            part.load_weights({local: None if (spec.optional and present is not None and not present(prefix + local))
                               else fetch(prefix + local) for local, spec in names.items()}, ops)
        if getattr(self.head, "tied", False):
            self.head.tie(self.embedding)

    def step_lists(self) -> list:
        """The host-built lists that the model's parts ask of every step, each name once."""
        found: dict = {}
        for _, part in self._named:
            for sl in part.step_lists():
                found.setdefault(sl.name, sl)
        return list(found.values())

    # ---- cache ---------------------------------------------------------------------------
    @property
    def embedding_slot(self):
        """The cache slot of an embedding that keeps something per request, else None."""
        return self.plan.num_cache_slots if hasattr(self.embedding, "cache_spec") else None

    def cache_keys(self) -> list[tuple[int, bool]]:
        """``(cache slot, writes)`` of every view that ``forward`` wants, each once."""
        keys = [(e.cache_slot, e.writes_cache) for e in self.plan.schedule]
        if self.embedding_slot is not None:
            keys.append((self.embedding_slot, True))
        return list(dict.fromkeys(keys))

    def cache_specs(self) -> list[PagedKVSpec | FixedStateSpec | None]:
        """What each cache slot of the schedule holds (from the mixer that writes it)."""
        specs: list = [None] * self.plan.num_cache_slots
        if self.embedding_slot is not None:      # an embedding that keeps something: a slot behind the layers'
            specs.append(self.embedding.cache_spec())
        for entry in self.plan.schedule:
            block = self.blocks[entry.layer]
            # a block that keeps something itself answers for its mixer too
            spec = block.cache_spec() if hasattr(block, "cache_spec") else block.mixer.cache_spec()
            if entry.writes_cache:
                specs[entry.cache_slot] = spec
            elif specs[entry.cache_slot] != spec:
                raise ValueError(
                    f"layer {entry.layer} reads cache slot {entry.cache_slot} holding "
                    f"{specs[entry.cache_slot]}, but needs {spec}")
        return specs

    # ---- forward -------------------------------------------------------------------------
    def forward(self, ops, step, cache_views: Mapping[tuple[int, bool], object]) -> torch.Tensor:
        step.scratch.clear()           # what kernels derived from the step in an earlier pass is stale
        x = torch.empty((step.num_tokens, self.plan.hidden_size), dtype=torch.float32,
                        device=step.token_ids.device)
        if self.embedding_slot is not None:
            self.embedding.forward(ops, step.token_ids, x, step, cache_views[(self.embedding_slot, True)])
        elif getattr(self.embedding, "wants_positions", False):
            self.embedding.forward(ops, step.token_ids, x, step.positions)
        else:
            self.embedding.forward(ops, step.token_ids, x)
        x0 = x.clone() if self.junction is not None else None      # the embedding output, for the junction
        for entry in self.plan.schedule:
            if entry.enter is not None:
                self.junction.forward(ops, x, x0, entry.enter, step)
            cache = cache_views[(entry.cache_slot, entry.writes_cache)]
            self.blocks[entry.layer].forward(ops, x, step, cache)
        ops.flush()                        # nothing a part asked for may still be held back
        if step.num_logit_rows == 0:
            return torch.empty((0, self.plan.vocab_size), dtype=torch.float32, device=x.device)
        h = self.final_norm.forward_rows(ops, x, step.logit_rows, step.act_dtype)
        return self.head.forward(ops, h)
