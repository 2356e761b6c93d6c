"""A model built from its description: parts with their weights, run in order.

Nothing here names an architecture.  ``Model`` builds every part the
description lists, loads the tensors they declare, and runs a step: embed,
the run entries in their order (each with the cache view of its entry; an embedding that keeps
something per request has the view behind theirs), then
the final norm and the head on the rows whose logits are wanted only (the
reference norms and multiplies the last row only,
engine/src/gpt2_gpu.cu:254-263).
"""

from __future__ import annotations

from ..parts.base import build_part, get_arrangement
from ..parts.spec import NoCache, PagedKV
from ..parts.streams import read_sum
from ..weights.loader import collect_specs, load_weights


class Model:
    def __init__(self, spec):
        self.spec = spec
        self.embedding = build_part(spec.embedding)
        self.position = build_part(spec.position) if spec.position is not None else None
        self.embedding_norm = build_part(spec.embedding_norm) if spec.embedding_norm is not None else None
        if self.embedding_norm is not None and not hasattr(self.embedding_norm, "normalize_in_place"):
            raise ValueError(f"the norm '{spec.embedding_norm.kind}' cannot norm the embedded tokens in place")
        self.layers = []
        for layer in spec.layers:
            arrangement = get_arrangement(layer.arrangement)
            missing = [role for role in arrangement.roles if role not in layer.parts]
            if missing:
                raise ValueError(f"arrangement '{layer.arrangement}' needs parts {missing}")
            self.layers.append((arrangement, {role: build_part(p) for role, p in layer.parts.items()}))
        self.final_norm = build_part(spec.final_norm)
        self.head = build_part(spec.head)
        # A step may be captured into a CUDA graph only if every part launches nothing but
        # kernels whose arguments stay valid from step to step; parts say so themselves.
        self.graph_safe = all(getattr(part, "graph_safe", False) for part in self.parts())
        # The step makes a work list of attention tiles only if some part says it reads one.
        self.wants_attention_tiles = any(getattr(part, "wants_attention_tiles", False) for part in self.parts())
        # A step of long portions may bring its work list as units of 256 tokens instead, if
        # every part that reads the list can read those too: then this is their number of heads
        # (the step shares long units among so many CTAs that heads x CTAs fill the GPU), else 0.
        heads = {getattr(part, "attention_unit_heads", 0) for part in self.parts() if getattr(part, "wants_attention_tiles", False)}
        self.attention_unit_heads = heads.pop() if len(heads) == 1 else 0

    def parts(self):
        found = [self.embedding]
        if self.position is not None:
            found.append(self.position)
        if self.embedding_norm is not None:
            found.append(self.embedding_norm)
        for _, parts in self.layers:
            found.extend(parts.values())
        found.extend([self.final_norm, self.head])
        return found

    def cache_needs(self):
        """What each run entry keeps per request: a need, or ``{role: need}`` when several parts of
        the layer keep something; None for an entry that keeps nothing or reads another's cache."""
        needs = []
        for entry in self.spec.order:
            arrangement, parts = self.layers[entry.layer]
            mine = {}
            for role in arrangement.cache_roles(parts):
                need = parts[role].cache_need()
                if isinstance(need, dict):
                    # a part that keeps several things (its own parts' needs, by name)
                    mine.update({f"{role}.{name}": one for name, one in need.items()})
                else:
                    mine[role] = need
            mine = {role: need for role, need in mine.items() if not isinstance(need, NoCache)}
            if entry.cache_of is not None:
                # the pages are the other entry's; state of a fixed size per request (a filter's last inputs) stays its own
                mine = {role: need for role, need in mine.items() if not isinstance(need, PagedKV)}
            if not mine:
                needs.append(None)
            elif (entry.cache_of is None and tuple(mine) == (arrangement.mixer_role(),)
                  and tuple(arrangement.cache_roles(parts)) == tuple(mine)):
                needs.append(mine[arrangement.mixer_role()])
            else:
                needs.append(mine)
        # an embedding that keeps something owns the entry behind the run entries
        if not isinstance(self.embedding.cache_need(), NoCache):
            needs.append(self.embedding.cache_need())
        return needs

    def load(self, model_dir: str, dtype, device, runtime=None):
        specs = collect_specs(self.parts())
        tensors = load_weights(model_dir, specs, dtype, device, self.spec.file_prefixes, self.spec.ignored_weights)
        for part in self.parts():
            part.bind({w.name: tensors[w.name] for w in part.weight_specs() if w.name in tensors}, runtime)
        self.weight_bytes = sum(t.numel() * t.element_size() for t in
                                {t.data_ptr(): t for t in tensors.values()}.values())
        return self

    def _first_norm(self, index):
        """The norm that reads the stream first in run entry ``index``, if its arrangement says so."""
        if index >= len(self.spec.order):
            return None
        arrangement, parts = self.layers[self.spec.order[index].layer]
        return parts.get(arrangement.first_norm) if arrangement.first_norm is not None else None

    def forward(self, ctx, cache_views):
        """Run the step's tokens; returns fp32 logits [n_want, vocab] or None."""
        kept = {"cache": cache_views[len(self.spec.order)]} if len(cache_views) > len(self.spec.order) else {}
        hidden = self.embedding.forward(ctx, self.position, **kept)
        if self.embedding_norm is not None:
            self.embedding_norm.normalize_in_place(ctx, hidden)
        ctx.kept_results = None
        if self.spec.keeps_layer_results:
            # the embedding output is result 0; every layer's "depth_mix" part stores its own
            ctx.kept_results = ctx.buffer("kept_results", (ctx.n_tokens, len(self.spec.order) + 1, self.spec.hidden_size),
                                          hidden.dtype)
            ctx.kernels.depth_mix(hidden, ctx.kept_results, None, 0)
        ctx.streams = ctx.streams_pending = None
        ctx.rounded_stream = None        # the stream's rows in the activations' type, where an arrangement keeps them
        if self.spec.residual_streams > 0:
            # several residual streams, all equal to the embedding output at the start
            ctx.streams = ctx.buffer("streams", (ctx.n_tokens, self.spec.residual_streams, self.spec.hidden_size), hidden.dtype)
            ctx.kernels.streams_fill(ctx.streams, hidden)
        dump = getattr(ctx, "dump", None)
        if dump is not None:
            dump.append(hidden.clone())
        ctx.normed_ahead = None          # (norm part, its rows) where the pass that changed the stream last applied the next norm
        for index, entry in enumerate(self.spec.order):
            arrangement, parts = self.layers[entry.layer]
            ctx.next_norm = self._first_norm(index + 1)
            arrangement.run(ctx, parts, hidden, cache_views[index])
            if dump is not None:
                if ctx.streams is not None:
                    read_sum(ctx, hidden)
                dump.append(hidden.clone())
        if ctx.n_want == 0:
            return None
        if ctx.streams is not None:
            read_sum(ctx, hidden)
        defer = getattr(self.final_norm, "can_defer", False) and getattr(self.head, "accepts_deferred_norm", False)
        rows = self.final_norm.forward(ctx, hidden, rows=ctx.want_rows, tag="final_norm",
                                       **({"defer": True} if defer else {}))
        return self.head.forward(ctx, rows)
