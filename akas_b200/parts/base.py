"""What every part is, and the registries that map a spec's ``kind`` to a part.

A part is a mixer, a feed-forward, a norm or a position encoding. It is built
from its spec alone (``Part(spec, runtime)``), says which tensors it wants
(``params()``), takes them (``load()``), and computes (``forward()``). No part
knows which model it is in: names of checkpoint tensors reach it through the
prefix that the block passes, and sizes through its spec.

Interfaces (duck-typed; these base classes only document and give defaults):

* Norm: ``params()``, ``load(get)``, ``forward(x, out_dtype=None, rows=None)``; optionally
  ``lazy(h, rows=None)`` -> ``Normed`` so that a following product may absorb it.
* PositionEncoding: ``prepare(ctx)`` once per step, ``tables(ctx)`` -> (cos, sin)
  for the fused rotary kernel, or ``apply(q, k, ctx)`` for any other encoding.
* Mixer: ``params()``, ``load(get)``, ``cache()`` -> the cache it needs (a
  ``PagedKVSpec``, a ``StateSpec`` or ``None``), ``forward(x, ctx, cache, residual,
  write)``.
* FeedForward: ``params()``, ``load(get)``, ``forward(x, ctx, residual)``.

A mixer or feed-forward that can multiply what it adds into a residual by a constant sets ``takes_residual_scale``; the
block then sets its ``residual_scale``.

``forward`` of a mixer or feed-forward gets the normed activations ``x`` ``[N, C]``
in the compute dtype and, when ``residual`` is given (float32 ``[N, C]``), returns
``residual + result`` in float32 (it may add in place; the fused kernels do).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, Optional, Tuple

import torch


@dataclass(frozen=True)
class Param:
    """A tensor a part wants from the checkpoint.

    ``role`` decides the dtype it is held in: a ``"matrix"`` is an operand of a
    matrix product and takes the compute dtype; a ``"vector"`` (norm weights,
    convolution taps, biases) is held in float32; ``"table"`` is an integer table
    held in int32. ``optional`` tensors may be absent from the checkpoint. ``mean``
    is the mean that the random-weights mode draws the tensor around (1 for norm
    weights). A size of -1 in ``shape`` is whatever the checkpoint has there (a size
    that the configuration file does not give); ``default`` then names the size
    that the random-weights mode uses.
    """

    shape: Tuple[int, ...]
    role: str = "matrix"
    optional: bool = False
    mean: float = 0.0
    default: Tuple[int, ...] = ()

    def fits(self, shape) -> bool:
        return len(shape) == len(self.shape) and all(a in (-1, b) for a, b in zip(self.shape, shape))

    def concrete(self) -> Tuple[int, ...]:
        """The shape with every free size replaced by its default."""
        if -1 in self.shape and len(self.default) != len(self.shape):
            raise ValueError(f"a tensor of shape {self.shape} has a free size and no default for it")
        return tuple(d if a == -1 else a for a, d in zip(self.shape, self.default or self.shape))


class PagedSpec:
    """What a mixer with per-token storage asks of the cache manager; a mixer returns an instance from ``cache()``.

    ``pools(page_size)`` names its pools and gives the shape of ONE page of each (``{"k": (kv_heads, page, head_dim),
    ...}``); the manager allocates ``[pages, *shape]`` per pool and hands them over as attributes of the view the
    mixer gets (``cache.k``). ``window``: how many of the latest tokens are ever read (None: all); pages behind the
    window are given back while the request runs. ``page_size``: tokens per page if the mixer needs a size of its own
    (None: the engine's). ``dtype``: None for the compute dtype. Layers whose specs agree in ``paging()`` share page
    numbers, a free list and a block table; everything else (what a page holds) is the layer's own."""

    window: Optional[int] = None
    page_size: Optional[int] = None
    dtype: Optional[torch.dtype] = None
    keep_first: int = 0  # with a window: the first keep_first tokens are read for ever, so their pages are never given back
    # with a window: tokens are read once more when the block of ``pool`` tokens they are in is complete, so a page stays
    # until the blocks it holds a part of are
    pool: int = 0

    def pools(self, page_size: int) -> Dict[str, Tuple[int, ...]]:
        raise NotImplementedError

    def paging(self) -> tuple:
        return (self.window, self.page_size, self.keep_first if self.window else 0, self.pool if self.window else 0)


@dataclass(frozen=True)
class PagedKVSpec(PagedSpec):
    """Keys and values of every position (or of the last ``window`` and the first ``keep_first``), in pages
    ``[kv_heads, page, head_dim]`` (values: ``v_head_dim`` where that is given)."""

    num_kv_heads: int = 1
    head_dim: int = 16
    window: Optional[int] = None
    page_size: Optional[int] = None
    dtype: Optional[torch.dtype] = None
    keep_first: int = 0
    v_head_dim: Optional[int] = None
    pool: int = 0

    def pools(self, page_size: int) -> Dict[str, Tuple[int, ...]]:
        return {"k": (self.num_kv_heads, page_size, self.head_dim),
                "v": (self.num_kv_heads, page_size, self.v_head_dim or self.head_dim)}


@dataclass(frozen=True)
class PagedBlocksSpec(PagedSpec):
    """One key and one value for every whole block of ``block`` tokens, for ever: a block lies in the page of its last
    token, so a page of ``page_size`` tokens holds at most ceil(page_size / block) of them, in their order:
    ``[kv_heads, ceil(page_size / block), head_dim]`` (values: ``v_head_dim``). Block b of a request is entry
    b - floor(first / block) of its page, with ``first`` the page's first position."""

    block: int = 16
    num_kv_heads: int = 1
    head_dim: int = 16
    v_head_dim: Optional[int] = None
    page_size: Optional[int] = None
    dtype: Optional[torch.dtype] = None

    def pools(self, page_size: int) -> Dict[str, Tuple[int, ...]]:
        entries = -(-page_size // self.block)
        return {"k": (self.num_kv_heads, entries, self.head_dim), "v": (self.num_kv_heads, entries, self.v_head_dim or self.head_dim)}


@dataclass(frozen=True)
class PagedLatentSpec(PagedSpec):
    """One row of ``width`` numbers per position (or per position of the last ``window``) that serves as key and,
    by its first channels, as value for every head: pages ``[1, page, width]`` in one pool, ``kv``."""

    width: int = 16
    window: Optional[int] = None
    page_size: Optional[int] = None
    dtype: Optional[torch.dtype] = None
    keep_first: int = 0

    def pools(self, page_size: int) -> Dict[str, Tuple[int, ...]]:
        return {"kv": (1, page_size, self.width)}


@dataclass(frozen=True)
class StateSpec:
    """Per-request state of fixed size: one row of ``shape`` per request slot, zero at admission."""

    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class Runtime:
    """What a part needs to know about where it runs: compute dtype, device, kernels."""

    dtype: torch.dtype
    device: torch.device
    ops: Any


class Normed:
    """The output of a norm that has not run yet: ``norm(h[rows])``.

    A block hands it to parts that set ``takes_normed``; they pass it to ``project`` /
    ``project_swiglu`` for their first matrix product, where the kernels may compute the norm inside
    the product instead of in a pass of its own. ``tensor()`` runs the norm and gives the plain result.
    """

    def __init__(self, norm, h, rows=None):
        self.norm, self.h, self.rows = norm, h, rows
        self._tensor = None
        self.partner: Optional["Normed"] = None  # another norm of the same rows, made with this one in one pass (norm_pair)
        self.absorbed = False  # a product has computed the norm on its way in: nobody wants the tensor

    def tensor(self):
        if self._tensor is None:
            other = self.partner
            if other is not None and other._tensor is None and not other.absorbed:
                spec = self.norm.spec
                self._tensor, other._tensor = self.norm.rt.ops.rmsnorm_pair(
                    self.h, self.norm.weight, other.norm.weight, spec.eps, spec.zero_centered, self.norm.rt.dtype)
            else:
                self._tensor = self.norm.forward(self.h, rows=self.rows)
        return self._tensor


def norm_pair(first, second, h):
    """Two norms of the same rows that have not run yet. Two RMSNorms with the same eps read the rows once where the
    operations offer that, unless a product takes one of them in."""
    a, b = Normed(first, h), Normed(second, h)
    sa, sb = first.spec, second.spec
    alike = all(getattr(sa, f, None) == getattr(sb, f, None) for f in ("kind", "eps", "zero_centered"))
    if alike and getattr(sa, "kind", None) == "rmsnorm" and hasattr(first.rt.ops, "rmsnorm_pair"):
        a.partner, b.partner = b, a
    return a, b


def project(rt: "Runtime", x, w, out_dtype=None, residual=None, bias=None):
    """``x . w^T`` for a tensor or a ``Normed``; with ``residual`` the product is added into it; ``bias`` (float32, one
    number per output channel) is added before the result is rounded."""
    if isinstance(x, Normed):
        spec = x.norm.spec
        kind = getattr(spec, "kind", None)
        if residual is None and bias is None and kind == "rmsnorm" and _takes_norm(rt.ops, x, w):
            x.absorbed = True
            return rt.ops.norm_linear(x.h, x.norm.weight, spec.eps, spec.zero_centered, w, out_dtype, x.rows)
        if residual is None and bias is None and kind == "dynamic_tanh" and hasattr(rt.ops, "dyt_linear"):
            out = rt.ops.dyt_linear(x.h, x.norm.alpha, x.norm.weight, x.norm.shift, w, out_dtype, x.rows)
            if out is not None:
                return out
        x = x.tensor()
    if bias is not None:
        return rt.ops.linear(x, w, out_dtype=out_dtype, residual=residual, bias=bias)
    return rt.ops.linear(x, w, out_dtype=out_dtype, residual=residual)


def _takes_norm(ops, x: Normed, w) -> bool:
    """Whether ``ops.norm_linear`` should have this norm: always for a norm that stands alone; one of a pair only where
    the product really computes it on its way in (else the pair's one pass is the cheaper way)."""
    if not hasattr(ops, "norm_linear"):
        return False
    return x._tensor is None and (x.partner is None or (hasattr(ops, "absorbs_norm") and ops.absorbs_norm(x.h, w)))


def project_gated(rt: "Runtime", x, w_gate_up, width, bias, activation):
    """``act(x . w_g^T + b_g) * (x . w_u^T + b_u)`` for the stacked ``[w_g; w_u]`` (``width`` rows each), for a tensor or a ``Normed``: in the
    read-out of the product where the kernels offer that, else the product in float32 and the activation's kernel."""
    ops = rt.ops
    if isinstance(x, Normed):
        if getattr(x.norm.spec, "kind", None) == "dynamic_tanh" and hasattr(ops, "dyt_linear"):
            out = ops.dyt_linear(x.h, x.norm.alpha, x.norm.weight, x.norm.shift, w_gate_up, None, x.rows, gated=(width, bias, activation))
            if out is not None:
                return out
        if getattr(x.norm.spec, "kind", None) == "rmsnorm" and hasattr(ops, "norm_linear_gated"):
            spec = x.norm.spec
            out = ops.norm_linear_gated(x.h, x.norm.weight, spec.eps, spec.zero_centered, w_gate_up, width, bias, activation, x.rows)
            if out is not None:
                x.absorbed = True
                return out
        x = x.tensor()
    if hasattr(ops, "linear_gated"):
        return ops.linear_gated(x, w_gate_up, width, bias, activation)
    return ops.gated_activation(ops.linear(x, w_gate_up, out_dtype=torch.float32), width, bias, activation, rt.dtype)


def project_swiglu(rt: "Runtime", x, w_gate_up):
    """``silu(x . w1^T) * (x . w3^T)`` for the stacked ``[w1; w3]``, for a tensor or a ``Normed``."""
    if isinstance(x, Normed):
        spec = x.norm.spec
        if getattr(spec, "kind", None) == "rmsnorm" and hasattr(rt.ops, "norm_linear"):
            return rt.ops.norm_linear(x.h, x.norm.weight, spec.eps, spec.zero_centered, w_gate_up, None, x.rows, True)
        x = x.tensor()
    if hasattr(rt.ops, "linear_swiglu"):
        return rt.ops.linear_swiglu(x, w_gate_up)
    return rt.ops.swiglu(rt.ops.linear(x, w_gate_up))


class Part:
    takes_normed = False  # True: forward accepts a ``Normed`` in place of the normed tensor
    # True: the part reads and writes device tensors through ``runtime.ops`` functions only, so an operations module
    # that defers launches (a decode step run as one chain) may keep deferring across it. A part that computes with
    # torch directly leaves this False, and the decoder makes everything pending run before the part does.
    chain_safe = False
    # True: the part adds ``residual_scale`` times its result into a residual (a constant that the block sets before
    # loading); a part that leaves this False is asked for its result and the block adds it.
    takes_residual_scale = False
    residual_scale = 1.0

    def __init__(self, spec, runtime: Runtime):
        self.spec = spec
        self.rt = runtime

    def params(self) -> Dict[str, Param]:
        return {}

    def load(self, get: Callable[[str], torch.Tensor]) -> None:
        pass


class Mixer(Part):
    # True: another entry of the run order may read this mixer's cache (``write=False``) after the owner has run in
    # the same step, and sees the same past however the tokens were cut into steps: attention does, since every
    # earlier token's keys and values lie in the cache by then. A mixer whose cache is a summary of the past leaves
    # this False: once the owner has run, the summary has moved past the step's tokens, so a reader would see another
    # past in a step of one token than in a step of many. The decoder refuses a run order that shares such a cache.
    shares_cache = False

    @classmethod
    def kernels(cls, spec) -> tuple:
        """The kinds of compiled kernels a mixer of this spec launches (keys of ``ops.cuda._PART_FILES``), so that a
        model's first call builds what it needs and nothing else. A mixer that names none uses the products only."""
        return ()

    def cache(self):
        return None

    def forward(self, x, ctx, cache=None, residual=None, write=True):
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x, ctx, residual=None):
        raise NotImplementedError


_REGISTRIES: Dict[str, Dict[str, type]] = {"mixer": {}, "ffn": {}, "norm": {}, "position": {}}


def _register(family: str, kind: str, cls: type) -> None:
    _REGISTRIES[family][kind] = cls


def register_mixer(kind: str, cls: type) -> None:
    _register("mixer", kind, cls)


def register_ffn(kind: str, cls: type) -> None:
    _register("ffn", kind, cls)


def register_norm(kind: str, cls: type) -> None:
    _register("norm", kind, cls)


def register_position(kind: str, cls: type) -> None:
    _register("position", kind, cls)


def mixer_class(spec) -> type:
    """The class registered for a mixer spec's kind."""
    kind = getattr(spec, "kind", None)
    if kind not in _REGISTRIES["mixer"]:
        raise KeyError(f"no mixer registered for kind {kind!r}; registered: {sorted(_REGISTRIES['mixer'])}")
    return _REGISTRIES["mixer"][kind]


def ffn_class(spec) -> type:
    """The class registered for a feed-forward spec's kind."""
    kind = getattr(spec, "kind", None)
    if kind not in _REGISTRIES["ffn"]:
        raise KeyError(f"no ffn registered for kind {kind!r}; registered: {sorted(_REGISTRIES['ffn'])}")
    return _REGISTRIES["ffn"][kind]


def build_part(family: str, spec, runtime: Runtime):
    """The part that ``spec.kind`` names in the registry of ``family``; ``None`` for a ``None`` spec."""
    if spec is None:
        return None
    table = _REGISTRIES[family]
    kind = getattr(spec, "kind", None)
    if kind not in table:
        raise KeyError(f"no {family} registered for kind {kind!r}; registered: {sorted(table)}")
    return table[kind](spec, runtime)


def norm_params(norm, name: str) -> Dict[str, Param]:
    """Checkpoint name -> Param for a norm whose weight a layer names whole (``name``). A norm with more tensors than
    its weight lists the weight first and the others under local names that start with a dot; they stand beside the
    weight as ``name + local``."""
    items = list(norm.params().items())
    out = {name: items[0][1]}
    for local, param in items[1:]:
        out[name + local] = param
    return out


def load_norm(norm, name: str, get: Callable[[str], torch.Tensor]) -> None:
    """Hands a norm its tensors from the names that ``norm_params`` gave them."""
    main = next(iter(norm.params()))
    norm.load(lambda local: get(name if local == main else name + local))


def stack_rows(matrices, multiple: int = 16) -> torch.Tensor:
    """Matrices [o_i, K] that multiply the same input, stacked into one [sum o_i rounded up to ``multiple``, K] (the
    added rows are zero), so that one product feeds them all and its rows have a pitch that every product kernel writes."""
    rows = sum(m.shape[0] for m in matrices)
    pad = -rows % multiple
    if pad:
        matrices = list(matrices) + [torch.zeros((pad, matrices[0].shape[1]), dtype=matrices[0].dtype, device=matrices[0].device)]
    return torch.cat(list(matrices), dim=0).contiguous()


def renamed(spec, local: str) -> str:
    """The checkpoint's name for a part's local parameter name (``spec.names`` overrides)."""
    names = getattr(spec, "names", None) or {}
    return names.get(local, local)
