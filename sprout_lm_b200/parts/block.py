"""Arrangements of a layer's parts.  ``pre_norm``: x += mixer(norm_0(x)); x += ffn(norm_1(x))
(src/qwen.ts:164-200); a layer without a feed-forward (``feed_forward.kind == "none"``) is the first half alone.
``options["branch_scale"]`` multiplies what both sublayers add: the parts take it as their ``out_scale`` and fold it into
a step they have anyway."""
from __future__ import annotations

from ..config.specs import LayerSpec, PartSpec
from .base import Part, build_part, register_part


def scaled(spec: PartSpec, factor: float) -> PartSpec:
    """The part with its output multiplied by ``factor`` (its ``out_scale`` parameter)."""
    if factor == 1.0:
        return spec
    return PartSpec(spec.kind, {**spec.params, "out_scale": factor * spec.params.get("out_scale", 1.0)})


@register_part("block", "pre_norm")
class PreNormBlock(Part):
    def __init__(self, prefix: str, layer: LayerSpec):
        self.has_ffn = layer.feed_forward.kind != "none"
        if len(layer.norms) != (2 if self.has_ffn else 1):
            raise ValueError("a pre_norm block has one norm per sublayer")
        self.norms = [build_part("norm", spec, prefix) for spec in layer.norms]
        branch = float(layer.options.get("branch_scale", 1.0))
        self.mixer = build_part("mixer", scaled(layer.mixer, branch), prefix)
        self.feed_forward = build_part("feed_forward", scaled(layer.feed_forward, branch), prefix) if self.has_ffn else None

    def parts(self):
        return [*self.norms, self.mixer, *([self.feed_forward] if self.has_ffn else [])]

    def tensor_decls(self):
        return [decl for part in self.parts() for decl in part.tensor_decls()]

    def load(self, source):
        for part in self.parts():
            part.load(source)

    def forward(self, x, ctx, cache, state):
        # a mixer or a feed-forward may offer to take the norm before it into its own kernel
        fused = getattr(self.mixer, "forward_with_norm", None)
        if fused is None or not fused(self.norms[0], x, ctx, cache, state):
            self.mixer.forward(self.norms[0].forward(x), x, ctx, cache, state)
        if not self.has_ffn:
            return
        fused = getattr(self.feed_forward, "forward_with_norm", None)
        if fused is None or not fused(self.norms[1], x, ctx):
            self.feed_forward.forward(self.norms[1].forward(x), x, ctx)


def build_block(layer: LayerSpec):
    from .base import _REGISTRY
    from ..config.specs import ConfigError
    try:
        cls = _REGISTRY["block"][layer.block]
    except KeyError:
        raise ConfigError(f"no block arrangement {layer.block!r} is registered") from None
    return cls(prefix=layer.prefix, layer=layer)


@register_part("block", "post_norm")
class PostNormBlock(Part):
    """The norm comes after the sum: x <- norm_0(alpha x + mixer(x)), then x <- norm_1(alpha x + ffn(x));
    the sublayers read x itself.  The sums and the stream are float32; a sublayer reads x in the compute
    dtype.  A layer without a feed-forward (``feed_forward.kind == "none"``) is the first half alone.

    A sublayer gets ``h`` = x in the compute dtype and ``y`` = alpha x (float32) and adds its output to
    y; the norm kernel that follows writes x and, for the second sublayer, the next h and y as well.
    """

    def __init__(self, prefix: str, layer: LayerSpec):
        self.alpha = float(layer.options.get("alpha", 1.0))
        self.has_ffn = layer.feed_forward.kind != "none"
        if len(layer.norms) != (2 if self.has_ffn else 1):
            raise ValueError("a post_norm block has one norm per sublayer")
        self.norms = [build_part("norm", spec, prefix) for spec in layer.norms]
        for norm in self.norms:
            if getattr(norm, "fused_kind", None) != "rmsnorm":
                raise ValueError("a post_norm block takes RMS norms")
        self.mixer = build_part("mixer", layer.mixer, prefix)
        self.feed_forward = build_part("feed_forward", layer.feed_forward, prefix) if self.has_ffn else None

    def parts(self):
        return [*self.norms, self.mixer, *([self.feed_forward] if self.has_ffn else [])]

    def tensor_decls(self):
        return [decl for part in self.parts() for decl in part.tensor_decls()]

    def load(self, source):
        for part in self.parts():
            part.load(source)
        self.dtype = source.runtime.dtype

    def readers(self, x):
        """Buffers for what this block's first sublayer reads: (y, h) with y = alpha x and h = x in the compute dtype
        (None in float32, where the sublayer reads x itself).  Whoever makes x may fill them (``primed``)."""
        import torch
        y = torch.empty_like(x)
        h = torch.empty(x.shape, dtype=self.dtype, device=x.device) if self.dtype != torch.float32 else None
        return y, h

    def forward(self, x, ctx, cache, state, primed=None, finish=None):
        """``primed``: (y, h) already filled for this x.  ``finish(y, gain, eps)``: instead of the block's last norm, the
        caller's continuation, which must leave the layer's result (or what follows from it) in x."""
        import torch
        from .. import kernels
        narrow = self.dtype != torch.float32
        if primed is None:
            y, h = self.readers(x)
            kernels.scale_cast(x, y, h, self.alpha)
        else:
            y, h = primed
        self.mixer.forward(h if narrow else x, y, ctx, cache, state)
        norm = self.norms[0]
        if self.has_ffn:
            kernels.sum_norm(y, norm.gain, x, norm.eps, y2=y, h=h, alpha=self.alpha)
            self.feed_forward.forward(h if narrow else x, y, ctx)
            norm = self.norms[1]
        if finish is not None:
            finish(y, norm.gain, norm.eps)
        else:
            kernels.sum_norm(y, norm.gain, x, norm.eps)


@register_part("block", "sandwich_norm")
class SandwichNormBlock(Part):
    """A norm before and after each sublayer: x += norm_1(mixer(norm_0(x))), then x += norm_3(ffn(norm_2(x))).
    The norms are layer norms or RMS norms, all of a block alike.
    The stream and the sums are float32.  A layer without a feed-forward (``feed_forward.kind == "none"``) has the
    first two norms only.  A sublayer adds its output into a zeroed float32 buffer; one kernel then norms that
    buffer, adds it to the stream, clears the buffer for the next sublayer and makes what that one reads.  That goes on
    from block to block: ``forward`` takes ``primed`` = (h, y), what the block before left (the first sublayer's input and
    the zeroed buffer), and returns the same for ``following``, the next block, or None."""
    chains = True

    def __init__(self, prefix: str, layer: LayerSpec):
        self.has_ffn = layer.feed_forward.kind != "none"
        if len(layer.norms) != (4 if self.has_ffn else 2):
            raise ValueError("a sandwich_norm block has two norms per sublayer")
        self.norms = [build_part("norm", spec, prefix) for spec in layer.norms]
        for norm in self.norms:
            if getattr(norm, "fused_kind", None) not in ("layernorm", "rmsnorm") or norm.fused_kind != self.norms[0].fused_kind:
                raise ValueError("a sandwich_norm block takes layer norms or RMS norms, all alike")
        self.rms = self.norms[0].fused_kind == "rmsnorm"
        self.mixer = build_part("mixer", layer.mixer, prefix)
        self.feed_forward = build_part("feed_forward", layer.feed_forward, prefix) if self.has_ffn else None

    def parts(self):
        return [*self.norms, self.mixer, *([self.feed_forward] if self.has_ffn else [])]

    def tensor_decls(self):
        return [decl for part in self.parts() for decl in part.tensor_decls()]

    def load(self, source):
        for part in self.parts():
            part.load(source)
        self.dtype = source.runtime.dtype

    def _close(self, y, x, after, following):
        """x += after(y); with a norm ``following`` y is cleared and that norm's output of the new x returned."""
        import torch
        from .. import kernels
        if following is None:
            kernels.norm_add(y, after.gain, x, after.eps, rms=self.rms)
            return None
        if following.eps != after.eps or getattr(following, "bias", None) is not None:
            kernels.norm_add(y, after.gain, x, after.eps, rms=self.rms, clear=True)
            return following.forward(x)
        h = torch.empty(x.shape, dtype=self.dtype, device=x.device)
        kernels.norm_add(y, after.gain, x, after.eps, next_gain=following.gain, h=h, rms=self.rms, clear=True)
        return h

    def forward(self, x, ctx, cache, state, primed=None, following=None):
        import torch
        h, y = primed if primed is not None else (self.norms[0].forward(x), torch.zeros_like(x))
        last = following.norms[0] if isinstance(following, SandwichNormBlock) and following.rms == self.rms else None
        self.mixer.forward(h, y, ctx, cache, state)
        if self.has_ffn:
            self.feed_forward.forward(self._close(y, x, self.norms[1], self.norms[2]), y, ctx)
        h = self._close(y, x, self.norms[-1], last)
        return None if h is None else (h, y)


@register_part("block", "parallel_residual")
class ParallelResidualBlock(Part):
    """One norm whose output both sublayers read: h = norm_0(x), x += mixer(h) + ffn(h).  A layer without a feed-forward
    (``feed_forward.kind == "none"``) adds the mixer alone.  ``options["side"]`` (a ``side_input`` PartSpec) runs after the
    sublayers and adds to the stream what it makes from the step's token ids.  The stream and the sum are float32."""

    def __init__(self, prefix: str, layer: LayerSpec):
        self.has_ffn = layer.feed_forward.kind != "none"
        if len(layer.norms) != 1:
            raise ValueError("a parallel_residual block has one norm")
        self.norms = [build_part("norm", layer.norms[0], prefix)]
        self.mixer = build_part("mixer", layer.mixer, prefix)
        self.feed_forward = build_part("feed_forward", layer.feed_forward, prefix) if self.has_ffn else None
        side = layer.options.get("side")
        self.side = build_part("side_input", side, prefix) if side is not None else None

    def parts(self):
        return [*self.norms, self.mixer, *([self.feed_forward] if self.has_ffn else []), *([self.side] if self.side else [])]

    def tensor_decls(self):
        return [decl for part in self.parts() for decl in part.tensor_decls()]

    def load(self, source):
        for part in self.parts():
            part.load(source)

    def forward(self, x, ctx, cache, state):
        h = self.norms[0].forward(x)
        self.mixer.forward(h, x, ctx, cache, state)
        if self.has_ffn:
            self.feed_forward.forward(h, x, ctx)
        if self.side is not None:
            self.side.forward(x, ctx)
