"""A whole model put together from a :class:`~alofa_b200.config.spec.ModelSpec`.

The run list is data: ``spec.run`` names, per position, which layer runs and
which cache it uses.  A layer named twice runs twice with the same weights; an
entry whose cache is an earlier entry's reads that cache and writes nothing
(layer order of the one shipped architecture: src/alofa/model/arch/qwen.mojo:1367-1372)."""
from __future__ import annotations

import numpy as np
import torch

from ..config.spec import ModelSpec
from ..csrc import ops
from ..errors import AlofaError
from .base import Runtime, build_part


class Model:
    def __init__(self, spec: ModelSpec, rt: Runtime):
        spec.validate()
        self.spec = spec
        self.rt = rt
        self.embedding = build_part("embedding", spec.embedding, rt)
        self.layers = [build_part("block", layer.block, rt) for layer in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, rt)
        self.head = build_part("head", spec.head, rt)
        self.run = [(e.layer, i if e.cache is None else e.cache) for i, e in enumerate(spec.run)]
        # per run entry: the norm that what follows starts with, where a block before it may make those rows (the final norm only when every row is wanted)
        norms = [getattr(self.layers[layer], "first_norm", None) for layer, _ in self.run[1:]] + [self.final_norm]
        self.next_norms = [n if n is not None and n.spec.kind == "rmsnorm" else None for n in norms]
        # a block may read the embedding output of the step's tokens later on (ctx.embedding_output)
        self.keeps_embedding = any(getattr(block, "needs_embedding_output", False) for block in self.layers)
        # whether a mixer goes another way in steps whose requests all start in them
        self.tells_fresh = any(getattr(getattr(block, "mixer", None), "tells_fresh", False) for block in self.layers)
        # blocks that keep several copies of the residual stream say how many (ctx.streams); every block of a model says the same
        # mixers that mix their values with those of the first of them: the values of a step's tokens are kept for it (ctx.first_values)
        widths = {int(getattr(block, "shared_value_width", 0)) for block in self.layers} - {0}
        if len(widths) > 1:
            raise AlofaError("unsupported", "layers that mix their values must have the same number of them", f"widths={sorted(widths)}")
        self.shared_value_width = widths.pop() if widths else 0
        copies = {int(getattr(block, "stream_copies", 0)) for block in self.layers}
        if len(copies) > 1:
            raise AlofaError("unsupported", "blocks over several residual streams cannot be mixed with others", f"stream_copies={sorted(copies)}")
        self.stream_copies = copies.pop() if copies else 0

    def parts(self):
        return [self.embedding, *self.layers, self.final_norm, self.head]

    def tensors(self) -> dict:
        out = {}
        for part in self.parts():
            out.update(part.tensors())
        return out

    def load(self, state: dict) -> None:
        state = dict(state)
        for part in self.parts():
            part.load(state)

    def graph_safe(self) -> bool:
        """True when every part may be recorded in a CUDA graph."""
        return all(part.graph_safe for part in self.parts())

    def scratch_row_bytes(self) -> tuple:
        """(bytes per token that live for a whole step, bytes per token of the
        layer that needs most): what the step runner sizes its arena from."""
        hidden = self.spec.hidden_size
        per_layer = max([getattr(block, "scratch_row_bytes", lambda: 0)() for block in self.layers] + [8 * hidden])
        return 4 * hidden + 4 * hidden + (4 * hidden if self.keeps_embedding else 0) + 4 * self.shared_value_width + (4 * hidden * self.stream_copies if self.stream_copies > 1 else 0), per_layer

    def cache_plan(self) -> dict:
        """run index -> cache spec, for the entries that own a cache."""
        return {i: self.layers[layer].cache_spec() for i, (layer, cache) in enumerate(self.run) if cache == i}

    def forward(self, ctx, caches: dict) -> torch.Tensor:
        """Logits (fp32) at ``ctx.logit_rows`` for the step's tokens (None when
        no row is wanted; the final norm and the head run on wanted rows only)."""
        h = ctx.buf((ctx.n_tokens, self.spec.hidden_size), torch.float32)
        ctx.stream_rows = None  # nothing is left over from another pass over the layers
        ctx.open_stream(h)
        self.embedding.forward(ctx, h)
        if self.keeps_embedding:
            ctx.embedding_output = ctx.buf(tuple(h.shape), torch.float32)
            ctx.embedding_output.copy_(h)
        if self.shared_value_width:
            ctx.first_values = ctx.buf((ctx.n_tokens, self.shared_value_width), torch.float32)
        if self.stream_copies:
            ctx.open_streams(h, self.stream_copies)
        # every row wanted, in order (a decode step): no picking, and the last block or a norm that reads the stream as base + accumulator may make them
        all_rows = ctx.n_out == ctx.n_tokens and bool((ctx.host_field("logit_rows") == np.arange(ctx.n_tokens, dtype=np.int32)).all())
        last = len(self.run) - 1
        for i, (layer, cache) in enumerate(self.run):
            block = self.layers[layer]
            if not getattr(block, "absorbs_pending", False):
                ctx.flush_pending()
            ctx.begin_layer()
            ctx.next_norm = self.next_norms[i] if i < last or all_rows else None
            block.forward(ctx, h, caches.get(cache), writes=(cache == i))
        ctx.end_layers()
        if self.stream_copies:
            ctx.sum_streams(h)
        if ctx.n_out == 0:  # a prompt portion whose logits nobody wants
            ctx.close_stream()
            return None
        if not getattr(self.final_norm, "absorbs_pending", False):
            ctx.flush_pending()
        left, ctx.stream_rows = ctx.stream_rows, None
        if all_rows and left is not None and left[0] is h and left[2] is self.final_norm:
            x = left[1]
        else:
            x = self.final_norm.forward(ctx, h, None if all_rows else ctx.logit_rows)
        ctx.close_stream()
        return self.head.forward(ctx, x)

def expected_tensors(spec: ModelSpec) -> dict:
    """name -> TensorSpec of everything the model reads from a checkpoint."""
    return Model(spec, Runtime(torch.device("cpu"), torch.float32)).tensors()
