"""A decoder put together from parts, as its ModelSpec says.

Reference forward (engine/model.py:280-299, 322-331): embedding, the layers,
final norm on the rows whose logits are wanted, output head.  Here the layers
are parts built from specs, and the order they run in is the spec's list.
"""

from __future__ import annotations

from typing import List, Optional

import torch

from ..config.registry import load_config
from ..parts.registry import build_part, part_class
from ..weights.loader import Checkpoint, WeightsError
from .context import ResidualStream, Runtime, StepContext, StreamResidual


class DecoderModel:
    def __init__(self, spec, names, checkpoint: Checkpoint, runtime: Runtime):
        checkpoint.check(spec, names)
        self.spec = spec
        self.runtime = runtime
        ops, dtype, device = runtime.ops, runtime.dtype, runtime.device

        def load(name):
            return checkpoint.load(name, dtype, device)

        self.embedding = load(names.embedding).contiguous()   # a table to gather rows from: no product reads it ...
        if checkpoint.has(names.lm_head):
            # engine/model.py:103-107: an lm_head in the file is used even when the config ties.
            self.lm_head = ops.prepare_matrix(load(names.lm_head))
        elif spec.tie_embeddings:
            self.lm_head = ops.prepare_matrix(self.embedding)   # ... unless it is the output head as well (same tensor)
        else:
            raise WeightsError(f"{checkpoint.where}: {names.lm_head} is missing and the embeddings are not tied")
        norm_cls = part_class("norm", spec.final_norm.kind)
        self.final_norm = norm_cls(spec.final_norm,
                                   {r: load(names.final_norm[r]) for r in norm_cls.weight_shapes(spec.final_norm)}, runtime)
        self.embedding_norm = None
        if getattr(spec, "embedding_norm", None) is not None:
            if not spec.residual_float32 or spec.streams is not None or spec.position_embedding is not None or spec.loop is not None \
                    or spec.embedding_scale is not None:
                raise ValueError("a norm of the embedded rows makes one 32-bit residual and nothing else enters there")
            self.embedding_norm = build_part("norm", spec.embedding_norm, {r: load(n) for r, n in names.embedding_norm.items()}, runtime)
        self.position = None   # a position part that enters at the embedding
        if getattr(spec, "position_embedding", None) is not None:
            self.position = build_part("position", spec.position_embedding, {}, runtime)
        self.blocks = []
        for block_spec, block_names in zip(spec.layers, names.layers):
            block_cls = part_class("block", block_spec.kind)
            weights = {}
            for part_name, category, sub in block_cls.sub_parts(block_spec):
                roles = part_class(category, sub.kind).weight_shapes(sub)
                weights[part_name] = {role: load(block_names[part_name][role]) for role in roles}
            self.blocks.append(block_cls(block_spec, weights, runtime))
        self.pass_starts, self.loop_steps = {}, None
        if getattr(spec, "loop", None) is not None:
            if not spec.residual_float32 or spec.streams is not None or self.position is not None:
                raise ValueError("layers that run in passes need one 32-bit residual and positions that enter in the mixers")
            self.pass_starts = spec.pass_starts()
            self.loop_steps = checkpoint.load(names.loop_step, torch.float32, device).float().contiguous()
        self.order = spec.execution_order()
        for i in self.order:
            if not 0 <= i < len(self.blocks):
                raise ValueError(f"the execution order names layer {i}; the model has {len(self.blocks)} layers")

    # ---- construction ------------------------------------------------------------------

    @classmethod
    def from_folder(cls, folder, runtime: Runtime) -> "DecoderModel":
        config = load_config(folder)
        checkpoint = Checkpoint.open(folder)
        if hasattr(config, "with_shapes"):   # an architecture some of whose sizes only the tensors' shapes give
            config = config.with_shapes(checkpoint.shapes())
        try:
            model = cls(config.model_spec(), config.tensor_names(), checkpoint, runtime)
        finally:
            checkpoint.close()
        model.config = config
        return model

    @classmethod
    def from_source(cls, config, source, runtime: Runtime, where: str = "weight source") -> "DecoderModel":
        model = cls(config.model_spec(), config.tensor_names(), Checkpoint(source, where), runtime)
        model.config = config
        return model

    def parts(self):
        """Every part object of the model: the final norm, each block, and what each block is made of."""
        yield self.final_norm
        if self.embedding_norm is not None:
            yield self.embedding_norm
        for block, block_spec in zip(self.blocks, self.spec.layers):
            yield block
            for name, _, _ in type(block).sub_parts(block_spec):
                part = getattr(block, name, None)
                if part is not None:
                    yield part
                    yield from getattr(part, "children", tuple)()   # a part made of parts (mixers side by side)

    # ---- cache -------------------------------------------------------------------------

    def cache_requests(self) -> List[object]:
        """What each entry of the execution order asks of the cache.  A layer that is named twice runs
        with the same weights but keeps a cache entry per occurrence (otherwise the second run would
        overwrite what the first run of a later step has to read).  A mixer that reads another layer's
        cache gets the entry of that layer's latest earlier occurrence."""
        from ..cache.cache import SharedRequest
        requests = []
        for pos, i in enumerate(self.order):
            req = self.blocks[i].cache_request()
            if isinstance(req, SharedRequest):
                earlier = [p for p in range(pos) if self.order[p] == req.layer]
                if not earlier:
                    raise ValueError(f"layer {i} reads the cache of layer {req.layer}, which has not run before it")
                req = SharedRequest(earlier[-1])
            requests.append(req)
        return requests

    def prepare(self, cache) -> None:
        """Size position tables and workspaces for the cache the model will run on."""
        for block in self.blocks:
            block.prepare(cache)

    # ---- forward -----------------------------------------------------------------------

    def hidden(self, ctx: StepContext, tokens: torch.Tensor):
        """Run the step's rows through every layer; returns the residual stream before the final norm."""
        if self.spec.streams is not None:   # 32-bit copies of the scaled embedding rows, side by side
            x = ctx.ops.embed_streams(tokens, self.embedding, ctx.status, self.spec.embedding_scale, self.spec.streams)
            stream = StreamResidual(x, self.spec.streams)
            for pos, i in enumerate(self.order):
                self.blocks[i].forward(ctx, stream, ctx.cache.layers[pos])
            return stream
        if self.embedding_norm is not None:
            x = self.embedding_norm.embed(ctx, tokens, self.embedding)   # normed 32-bit rows
        elif self.position is not None:
            x = self.position.embed(ctx, tokens, self.embedding)   # 32-bit rows with the positions' vectors added
        elif self.spec.residual_float32 and self.spec.embedding_scale is not None:
            x = ctx.ops.embed_streams(tokens, self.embedding, ctx.status, self.spec.embedding_scale, 1)   # 32-bit rows, scaled
        elif self.spec.residual_float32 and self.embedding.dtype != torch.float32:
            x = ctx.ops.embed(tokens, self.embedding, ctx.status, out_float32=True)   # the residual stays 32-bit
        else:
            x = ctx.ops.embed(tokens, self.embedding, ctx.status)
        if self.spec.embedding_scale is not None and not self.spec.residual_float32:
            x = (x.float() * self.spec.embedding_scale).to(x.dtype)
        if self.pass_starts:
            return self._hidden_in_passes(ctx, x)
        stream = ResidualStream(x)
        for pos, i in enumerate(self.order):
            self.blocks[i].forward(ctx, stream, ctx.cache.layers[pos])
        return stream

    def _hidden_in_passes(self, ctx: StepContext, embedded: torch.Tensor):
        """The layers of a model with a loop: before a pass's first layer the residual takes the embedding output (every
        pass but the first) and the pass's own vector, in 32-bit.  The layers change the residual in place, so the
        embedding output is kept apart: the first sum is written to a new tensor."""
        ops = ctx.ops
        x = None if 0 in self.pass_starts else ops.add_rows(embedded)   # layers before the loop work on a copy
        stream = ResidualStream(x)
        for pos, i in enumerate(self.order):
            t = self.pass_starts.get(pos)
            if t is not None:
                if stream.x is None:
                    stream.x = ops.add_rows(embedded, None, self.loop_steps[t])
                else:
                    ops.add_rows(stream.x, embedded if t > 0 else None, self.loop_steps[t], out=stream.x)
            self.blocks[i].forward(ctx, stream, ctx.cache.layers[pos])
        return stream

    def logits(self, ctx: StepContext, stream: ResidualStream, rows: Optional[torch.Tensor]) -> torch.Tensor:
        """32-bit logits [len(rows), vocab] at the given rows (all rows when None)."""
        ops = ctx.ops
        if rows is not None:
            stream = stream.at_rows(ops, rows)
        h = stream.normed(self.final_norm)   # takes what still waits on the stream first
        logits = ops.linear(h, self.lm_head, out_float32=True)
        if self.spec.logit_scale is not None:
            logits = logits * self.spec.logit_scale
        if self.spec.logit_softcap is not None:
            logits = ops.softcap(logits, self.spec.logit_softcap)
        return logits
