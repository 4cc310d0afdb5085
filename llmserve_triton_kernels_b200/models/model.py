"""A runnable model built from a :class:`ModelPlan`: the same class for every architecture.

It owns the token table, the layers (blocks of parts), the final norm and the output matrix,
declares every tensor it expects by checkpoint name, and runs one step over a flat batch of
tokens.  Parity for the order of operations: src/llmserve/model/llama.py:155-185 (embedding,
the layers in order, gather of the wanted rows *before* the final norm, output matrix).
"""

from __future__ import annotations

import torch

from .. import ops
from ..parts.base import Block, CompositeSpec, PagedKVSpec, PagedRowSpec, StateSpec, TensorSpec, build_part, part_factory
from .plan import ModelPlan


class Model:
    def __init__(self, plan: ModelPlan, dtype: torch.dtype, device: torch.device | str):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"compute dtype must be bfloat16 or float32, got {dtype}")
        self.plan = plan
        self.dtype = dtype
        self.device = torch.device(device)
        self.blocks: list[Block] = []
        self._named_parts: list[tuple[str, object]] = []  # (prefix, part) of every tensor-owning part
        for i, spec in enumerate(plan.layers):
            factory = part_factory("block", spec.block.kind)
            roles = getattr(factory, "roles", None)
            if not roles:
                raise ValueError(f"block kind {spec.block.kind!r} declares no roles (Block.roles: role -> part category)")
            if set(roles) != set(spec.parts):
                raise ValueError(
                    f"layer {i}: block kind {spec.block.kind!r} is built from {sorted(roles)}, the plan gives {sorted(spec.parts)}"
                )
            parts = {}
            for role, category in roles.items():
                parts[role] = build_part(category, spec.parts[role])
                self._named_parts.append((spec.parts[role].prefix, parts[role]))
            block = build_part("block", spec.block, **parts)
            self._named_parts.append((spec.block.prefix, block))
            self.blocks.append(block)
        self.final_norm = build_part("norm", plan.final_norm)
        self._named_parts.append((plan.final_norm.prefix, self.final_norm))
        self.embedding: torch.Tensor | None = None
        self.head: torch.Tensor | None = None
        self.position_table: torch.Tensor | None = None
        self._injections = {inj.before: inj for inj in plan.injections}
        self._vectors: dict[str, torch.Tensor] = {}  # the plan's extra tensors, 32-bit
        # a function (entry index, residual stream [N, hidden] with everything added) that is called after every
        # entry of the order when it is set: for looking at the stream layer by layer (it costs a copy per layer)
        self.layer_probe = None

    # ------------------------------------------------------------------ tensors
    def tensor_specs(self) -> dict[str, TensorSpec]:
        """Every tensor of the checkpoint by its full name."""
        plan = self.plan
        specs = {plan.embedding: TensorSpec((plan.vocab_size, plan.hidden_size))}
        if plan.positions is not None:
            specs[plan.positions] = TensorSpec((plan.max_positions, plan.hidden_size))
        for prefix, part in self._named_parts:
            for local, spec in part.tensors().items():
                name = prefix + local
                if name in specs:
                    raise ValueError(f"two parts claim the tensor {name!r}")
                specs[name] = spec
        if plan.head is not None:
            specs[plan.head] = TensorSpec((plan.vocab_size, plan.hidden_size))
        for name, shape in plan.extra_tensors:
            if name in specs:
                raise ValueError(f"two owners claim the tensor {name!r}")
            specs[name] = TensorSpec(tuple(shape))
        return specs

    def ignored_tensor_names(self) -> set[str]:
        """Names a checkpoint may carry that the model does not read; the plan lists them."""
        return set(self.plan.ignored)

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        plan = self.plan
        self.embedding = tensors[plan.embedding].to(device=self.device, dtype=self.dtype).contiguous()
        if plan.positions is not None:
            self.position_table = tensors[plan.positions].to(device=self.device, dtype=self.dtype).contiguous()
        if plan.head is None:
            self.head = self.embedding
        else:
            self.head = tensors[plan.head].to(device=self.device, dtype=self.dtype).contiguous()
        for prefix, part in self._named_parts:
            local = {name: tensors[prefix + name] for name in part.tensors()}
            part.bind(local, self.dtype, self.device)
        for name, _ in plan.extra_tensors:
            self._vectors[name] = tensors[name].to(device=self.device, dtype=torch.float32).contiguous()

    def weight_bytes(self) -> int:
        """Bytes of every distinct weight tensor a step reads (the token table only if it is also the head)."""
        seen: dict[int, int] = {}

        def visit(obj):
            for value in vars(obj).values():
                if isinstance(value, torch.Tensor):
                    seen[value.data_ptr()] = value.numel() * value.element_size()
                elif hasattr(value, "bind") and hasattr(value, "tensors"):
                    visit(value)

        for _, part in self._named_parts:
            visit(part)
        seen[self.head.data_ptr()] = self.head.numel() * self.head.element_size()
        return sum(seen.values())

    @property
    def graph_safe(self) -> bool:
        """Every part launches the same kernels whatever the step's contents, so a decode step can be captured."""
        return all(
            getattr(b, "graph_safe", False) for b in self.blocks
        ) and getattr(self.final_norm, "graph_safe", False)

    # ------------------------------------------------------------------ caches
    def cache_specs(self) -> list[PagedKVSpec | PagedRowSpec | StateSpec | CompositeSpec | None]:
        """For each entry of the order: what its mixer keeps, or None if it keeps nothing of its
        own (no cache, or it reads an earlier entry's)."""
        out = []
        for run in self.plan.schedule:
            out.append(None if run.cache_of is not None else self.blocks[run.layer].cache_spec())
        return out

    # ------------------------------------------------------------------ step
    def forward(self, ctx, caches) -> torch.Tensor:
        """Run the tokens of ``ctx`` through every entry of the order; ``caches[i]`` is the view
        of entry i's cache.  Returns 32-bit logits ``[len(ctx.logit_rows), vocab]``."""
        if ops.checked():
            self._check_step(ctx, caches)
        shared = getattr(ctx, "shared", None)
        if shared is not None:
            shared.clear()  # nothing of an earlier pass over this context is handed on
        resid, pending = self.embed_tokens(ctx), None
        if isinstance(resid, tuple):
            resid, pending = resid
        order = self.plan.schedule
        for i, run in enumerate(order):
            if i in self._injections:
                pending = self._inject(self._injections[i], resid, pending, ctx)
            # the norm that meets the stream next, so that a block's last product may prepare for it; none where
            # the stream takes something up in between: the contribution then comes back as it is
            follows = i + 1 < len(order) and (i + 1) not in self._injections
            next_norm = self.blocks[order[i + 1].layer].first_norm() if follows else None
            pending = self.blocks[run.layer].forward(resid, pending, ctx, caches[i], next_norm=next_norm)
            if self.layer_probe is not None:
                if isinstance(pending, ops.StreamUpdate):
                    self.layer_probe(i, self._updated_copies(resid, pending).sum(0))
                    continue
                delta, alpha = (None, 1.0) if isinstance(pending, ops.NormedInput) else ops.split_pending(pending)
                self.layer_probe(i, resid if delta is None else resid + alpha * delta.to(resid.dtype))
        if ctx.num_logits == 0:
            return torch.empty((0, self.plan.vocab_size), dtype=torch.float32, device=self.device)
        if self.plan.streams is not None:
            # the copies take up the last part's result and are summed, on the wanted rows only, in the final norm's kernel
            update = pending if isinstance(pending, ops.StreamUpdate) else None
            return self.project_logits(self.final_norm.add_streams(resid, update, None, rows=ctx.logit_rows))
        delta, alpha = ops.split_pending(pending)
        if alpha != 1.0:
            x = self.final_norm.add_forward(resid, delta, rows=ctx.logit_rows, alpha=alpha)
        else:
            x = self.final_norm.add_forward(resid, delta, rows=ctx.logit_rows)
        return self.project_logits(x)

    @staticmethod
    def _updated_copies(resid, update):
        """For looking at the stream only: the copies as they will be once ``update`` has been taken up (a new tensor)."""
        tensors, factors = update.results()
        y = sum(f * t.float() for t, f in zip(tensors, factors))
        return torch.einsum("st,snw->tnw", update.mix.view(resid.shape[0], resid.shape[0]), resid) + update.take.view(-1, 1, 1) * y[None]

    def _inject(self, inj, resid, pending, ctx):
        """The stream takes up what the entry in front left, then the token embeddings and/or a vector of the plan."""
        delta, alpha = ops.split_pending(pending)
        vector = self._vectors[inj.vector][inj.row] if inj.vector is not None else None
        if inj.add_embedding:
            ops.stream_inject(resid, delta, alpha, ctx.token_ids, self.embedding, vector)
        else:
            ops.stream_inject(resid, delta, alpha, None, None, vector)
        return None

    def _check_step(self, ctx, caches) -> None:
        """Checked mode: the step's arrays are looked over on the device before any kernel indexes with them."""
        from ..cache.manager import leaf_views

        caches = [leaf for c in caches for leaf in leaf_views(c)]
        slots = next((c.states.shape[0] for c in caches if hasattr(c, "states")), 0)
        ops.check_step_arrays(ctx, self.plan.vocab_size, self.plan.max_positions or 0x7FFFFFFF, slots)
        seen = []
        for c in caches:
            if hasattr(c, "page_table") and all(c.page_table.data_ptr() != t.data_ptr() for t in seen):
                ops.check_page_group(ctx, c.page_table, c.slot_map, c.page_size, c.pool.shape[0], c.spec.window, len(seen))
                seen.append(c.page_table)

    def embed_tokens(self, ctx) -> torch.Tensor:
        """The residual stream that the first layer meets: the tokens' rows of the table, in 32-bit ``[N, hidden]``.
        An architecture that scales or otherwise prepares its embeddings overrides this in a subclass that it names
        when it registers (``register_architecture(..., model_class=...)``).  May return a pair: the stream, and what the
        first block takes as pending (the same rows in the compute type, ``ops.StreamCopy``)."""
        if self.plan.streams is not None:
            x = ops.embed(ctx.token_ids, self.embedding, copies=self.plan.streams)  # [streams, N, hidden]
            if self.plan.embedding_scale != 1.0:
                ops.unary(x.view(-1, x.shape[-1]), "scale", self.plan.embedding_scale, inplace=True)
            return x
        if self.position_table is not None:
            wants_copy = self.dtype != torch.float32 and 0 not in self._injections and self.blocks[self.plan.schedule[0].layer].reads_stream
            x, copy = ops.embed_positions(ctx.token_ids, self.embedding, ctx.positions, self.position_table, self.plan.embedding_scale,
                                          copy_dtype=self.dtype if wants_copy else None)
            return x if copy is None else (x, ops.StreamCopy(copy))
        x = ops.embed(ctx.token_ids, self.embedding)
        if self.plan.embedding_scale != 1.0:
            ops.unary(x, "scale", self.plan.embedding_scale, inplace=True)
        return x

    def project_logits(self, x) -> torch.Tensor:
        """32-bit logits ``[rows, vocab]`` of the normalised rows ``x`` (a tensor, or the factored form that the
        last block handed on).  The place for an architecture's cap or scale of its logits, in a subclass."""
        logits = ops.linear(x, self.head, out_dtype=torch.float32)
        if self.plan.logit_scale != 1.0:
            ops.unary(logits, "scale", self.plan.logit_scale, inplace=True)
        if self.plan.logit_softcap is not None:
            ops.unary(logits, "softcap", self.plan.logit_softcap, inplace=True)
        return logits
