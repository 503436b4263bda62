"""Pre-norm block: `x += mixer(norm1(x)); x += ffn(norm2(x))`; a layer without a feed-forward has only the first half.

The sublayer outputs are not added at once: each norm adds the pending term of the sublayer before it, in one pass
over the row (fusezap/serve/models/llama.py:568, 600, 606: `x, h = add_norm(x, d, ln)`), and the model adds the last
one before the final norm (llama.py:608, 755).

Sandwich block: `x += post1(mixer(norm1(x))); x += post2(ffn(norm2(x)))`; the pending term carries its own norm.
"""
from __future__ import annotations
from dataclasses import replace
from ..weights import ParamSpec
from .base import Block, FeedForward, LayerCache, Mixer, Norm, PendingNorm, register_block


@register_block("pre_norm")
class PreNormBlock(Block):
    def __init__(self, mixer: Mixer, ffn: FeedForward | None, make_norm,
                 names: tuple[str, str, str, str] = ("input_layernorm", "self_attn", "post_attention_layernorm", "mlp"),
                 norms: tuple = (None, None)):
        """mixer, ffn: the layer's built parts; make_norm(spec): builds a norm. `norms`: a PartSpec for the norm before
        the mixer and one for the norm before the feed-forward (None: the layer's fallback kind), so the two may be of
        different kinds."""
        self.mixer, self.ffn, self.names = mixer, ffn, tuple(names)
        self.norm1 = make_norm(norms[0]) if norms[0] is not None else make_norm()
        self.norm2 = None
        if ffn is not None:
            self.norm2 = make_norm(norms[1]) if norms[1] is not None else make_norm()

    def children(self):
        n1, mx, n2, ff = self.names
        if self.ffn is None:
            return ((n1, self.norm1), (mx, self.mixer))
        return ((n1, self.norm1), (mx, self.mixer), (n2, self.norm2), (ff, self.ffn))

    def tensors(self) -> dict[str, ParamSpec]:
        # (a part whose tensor has the empty name owns the tensor called like its prefix)
        out = {(f"{prefix}.{k}" if k else prefix): v for prefix, part in self.children() for k, v in part.tensors().items()}
        if self.ffn is None:      # the second norm of an absent feed-forward is passed over if a checkpoint carries it
            for k, v in self.norm1.tensors().items():
                name = f"{self.names[2]}.{k}" if k else self.names[2]
                out[name] = replace(v, ignore=True)
        return out

    def bind(self, tensors, ops) -> None:
        for prefix, part in self.children():
            own = {k[len(prefix) + 1:]: v for k, v in tensors.items() if k == prefix or k.startswith(prefix + ".")}
            part.bind(own, ops)

    def forward(self, ctx, x, delta, cache: LayerCache):
        h = self.norm1.forward(ctx, x, delta)
        delta = self.mixer.forward(ctx, h, cache)
        if self.ffn is None:
            return x, delta
        h = self.norm2.forward(ctx, x, delta)
        delta = self.ffn.forward(ctx, h)
        return x, delta


@register_block("sandwich_norm")
class SandwichNormBlock(Block):
    """`x += post1(mixer(norm1(x))); x += post2(ffn(norm2(x)))`; a layer without a feed-forward has only the first half. A
    sublayer's result stays pending together with the norm it passes (`PendingNorm`), so that the next norm of the stream
    can norm it, add it and norm the sum in one pass over the row."""
    def __init__(self, mixer: Mixer, ffn: FeedForward | None, make_norm,
                 names: tuple = ("norm1", "mixer", "post1", "norm2", "ffn", "post2"), norms: tuple = (None, None, None, None)):
        """names: tensor-name prefixes of the norm before the mixer, the mixer, the norm after it, and the same three of the
        feed-forward. norms: PartSpecs of the four norms in that order (None: the layer's fallback kind)."""
        self.mixer, self.ffn, self.names = mixer, ffn, tuple(names)
        made = [make_norm(s) if s is not None else make_norm() for s in (norms if ffn is not None else norms[:2])]
        self.norm1, self.post1 = made[:2]
        self.norm2, self.post2 = made[2:] if ffn is not None else (None, None)

    def children(self):
        parts = (self.norm1, self.mixer, self.post1, self.norm2, self.ffn, self.post2)
        return tuple((n, p) for n, p in zip(self.names, parts) if p is not None)

    def tensors(self) -> dict[str, ParamSpec]:
        out = {(f"{prefix}.{k}" if k else prefix): v for prefix, part in self.children() for k, v in part.tensors().items()}
        if self.ffn is None:      # the norms of an absent feed-forward are passed over if a checkpoint carries them
            for name, norm in ((self.names[3], self.norm1), (self.names[5], self.post1)):
                out.update({(f"{name}.{k}" if k else name): replace(v, ignore=True) for k, v in norm.tensors().items()})
        return out

    def bind(self, tensors, ops) -> None:
        for prefix, part in self.children():
            part.bind({k[len(prefix) + 1:]: v for k, v in tensors.items() if k == prefix or k.startswith(prefix + ".")}, ops)

    def forward(self, ctx, x, delta, cache: LayerCache):
        h = self.norm1.forward(ctx, x, delta)
        delta = PendingNorm(self.mixer.forward(ctx, h, cache), self.post1)
        if self.ffn is None:
            return x, delta
        h = self.norm2.forward(ctx, x, delta)
        return x, PendingNorm(self.ffn.forward(ctx, h), self.post2)
