"""A model built from a plan: parts are looked up in the registries by kind,
given their params, and bound to the tensors the plan names.  The forward pass
walks the plan's running order; nothing here knows an architecture."""
import torch

from ..parts.registry import get_part
from ..weights.loader import DeviceStore, load_checked


def _as_tuple(need):
    return () if need is None else tuple(need) if isinstance(need, (tuple, list)) else (need,)


class Layer:
    """A built layer: `block` and the built sub-parts as attributes named by their roles."""

    def __init__(self, name, block, parts, mixer_role):
        self.name, self.block, self.parts = name, block, parts
        self.mixer_role = mixer_role
        self._spans = None
        for role, part in parts.items():
            setattr(self, role, part)

    @property
    def the_mixer(self):
        return self.parts[self.mixer_role] if self.mixer_role is not None else None

    def cache_need(self):
        """What a call of this layer keeps: the mixer's need as it is, or, where other sub-parts keep
        something too, one tuple of the mixer's needs followed by theirs in the order of the roles."""
        need = self.the_mixer.cache_need() if self.the_mixer is not None else None
        others = [p.cache_need() for role, p in self.parts.items() if role != self.mixer_role]
        others = [n for n in others if n is not None]
        if not others:
            return need
        return _as_tuple(need) + tuple(n for o in others for n in _as_tuple(o))

    def bindings(self, cache):
        """role -> its binding(s), of what cache_need() asked for (a block with a sub-part beside the
        mixer that keeps something takes its layer's cache apart with this)."""
        if self._spans is None:
            self._spans = self._make_spans()
        if self._spans == self.mixer_role:
            return {self.mixer_role: cache}
        return {role: cache[at] for role, at in self._spans}

    def _make_spans(self):
        """[(role, its place in the layer's tuple: an index, or a slice)]; the mixer's role alone where
        only the mixer keeps something."""
        roles = ([self.mixer_role] if self.mixer_role is not None else []) + \
            [r for r in self.parts if r != self.mixer_role]
        asked = [(r, self.parts[r].cache_need()) for r in roles]
        asked = [(r, n) for r, n in asked if n is not None]
        if len(asked) == 1 and asked[0][0] == self.mixer_role:
            return self.mixer_role
        spans, k = [], 0
        for role, need in asked:
            n = len(_as_tuple(need))
            spans.append((role, slice(k, k + n) if isinstance(need, (tuple, list)) else k))
            k += n
        return spans


class Model:
    def __init__(self, plan, runtime):
        self.plan = plan
        self.rt = runtime
        mk = lambda cat, spec: get_part(cat, spec.kind)(spec.params, runtime)
        self.embedding = mk("embedding", plan.embedding)
        self.position = mk("position", plan.position)
        self.layers = [Layer(lp.name, mk("block", lp.block),
                             {role: mk(cat, spec) for role, (cat, spec) in lp.parts.items()}, lp.mixer_role())
                       for lp in plan.layers]
        self.entries = [mk("stream_mix", spec) for spec in plan.entries]
        self.final_norm = mk("norm", plan.final_norm)
        self.head = mk("head", plan.head)
        for i, call in enumerate(plan.order):
            if not (0 <= call.layer < len(self.layers)):
                raise ValueError(f"running order entry {i} names layer {call.layer}, which does not exist")
            if call.cache_of is not None and not (0 <= call.cache_of < i):
                raise ValueError(f"running order entry {i} reads the cache of entry {call.cache_of}, "
                                 "which must come earlier")
            if call.enter is not None and not (0 <= call.enter[0] < len(self.entries)):
                raise ValueError(f"running order entry {i} names entry part {call.enter[0]}, which does not exist")
        self.weight_bytes = 0
        # a part that reads per-step host values (not only device arrays) cannot be replayed
        parts = [self.embedding, self.position, self.final_norm, self.head] + self.entries
        for layer in self.layers:
            parts += [layer.block] + list(layer.parts.values())
        self.graph_safe = all(getattr(p, "graph_safe", True) for p in parts)
        self.largest_layer_matrix = 0     # elements of the largest matrix a layer holds (set by load)

    def load(self, model_dir):
        refs = load_checked(self.plan, model_dir)
        store = DeviceStore(self.rt)
        pairs = [(self.embedding, self.plan.embedding), (self.position, self.plan.position)]
        n_head = len(pairs)
        for layer, lp in zip(self.layers, self.plan.layers):
            pairs += [(layer.parts[role], spec) for role, (_, spec) in lp.parts.items()]
        n_layers_end = len(pairs)
        pairs += list(zip(self.entries, self.plan.entries))
        pairs += [(self.final_norm, self.plan.final_norm), (self.head, self.plan.head)]
        for i, (part, spec) in enumerate(pairs):
            store.in_layer = n_head <= i < n_layers_end
            part.load({role: refs[name] for role, name in spec.weights.items()}, store)
        self.weight_bytes = store.bytes
        self.largest_layer_matrix = store.largest_layer_matrix
        return self

    def cache_needs(self):
        """(need per call of the running order, cache_of per call)."""
        needs = [self.layers[c.layer].cache_need() for c in self.plan.order]
        return needs, [c.cache_of for c in self.plan.order]

    def workspace_per_token(self):
        """Bytes of step workspace a token needs: the 32-bit residual stream, the widest layer (as
        its block says), and the final norm's rows."""
        E = self.plan.hidden_size
        act = 4 if self.rt.dtype == "float32" else 2
        blocks = [layer.block.workspace_per_token(layer) for layer in self.layers]
        return 4 * E + max(blocks + [0]) + act * E + sum(p.workspace_per_token() for p in self.entries)

    def graph_bound(self, ctx):
        """The upper bound of the context length that this step's kernels are launched for (a
        captured graph serves until the contexts pass it): the next power of two, unless a mixer
        asks for a tighter one."""
        bound = 128
        while bound < ctx.max_keys:
            bound *= 2
        asked = [b for b in (layer.the_mixer.graph_bound(ctx) for layer in self.layers
                             if layer.the_mixer is not None) if b is not None]
        if asked:
            bound = max(asked)
        return min(bound, self.plan.max_positions)

    def forward(self, ctx, cache, logits_out):
        """Run the step's tokens through every call of the running order; write
        the logits of the wanted rows into logits_out[:n_want]."""
        E = self.plan.hidden_size
        x = ctx.alloc((ctx.T, E), torch.float32)          # the residual stream, 32-bit
        self.embedding.forward(ctx, x, self.position)
        for part in self.entries:
            part.start(ctx, x)
        for i, call in enumerate(self.plan.order):
            layer = self.layers[call.layer]
            if call.enter is not None:
                self.entries[call.enter[0]].enter(ctx, x, call.enter[1])
            layer.block.forward(ctx, x, layer, cache.binding(i), self.position)
        if ctx.n_want > 0:
            for part in self.entries:
                part.close(ctx, x, ctx.want_rows)
            hf = ctx.alloc((ctx.n_want, E), self.rt.act_dtype)
            self.final_norm.forward(ctx, x, hf, rows=ctx.want_rows)
            self.head.forward(ctx, hf, logits_out[:ctx.n_want])
        return logits_out[:ctx.n_want]
