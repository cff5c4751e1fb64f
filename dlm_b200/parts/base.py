"""Interfaces of the parts a model is put together from.

A *part* has its sizes and constants as constructor parameters and never
learns which model it is in.  It names its tensors relative to itself
(``q_proj.weight``); the model prefixes them.  Four kinds of part exist:

* ``Norm``              ``forward(x_f32, rt, rows=None, out_dtype=None) -> activations``
* ``PositionEncoding``  gives the rotation table the attention kernels apply
* ``Mixer``             ``forward(h, resid, ctx, call)``: adds its output to ``resid``
* ``FeedForward``       ``forward(h, resid, ctx, pre_norm)``: adds its output to ``resid``

and a ``Block`` arranges one mixer, one feed-forward and their norms.

The residual stream ``resid`` is always 32-bit; ``h`` has the runtime's
activation dtype.  A mixer states what it needs cached through
``cache_need()`` (paged keys and values) and ``state_need()`` (a tensor of
fixed size per request); the cache manager groups equal needs.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable

import torch


@dataclass(frozen=True)
class ParamSpec:
    """One tensor a part reads.  ``init`` says how the random-weights mode draws it:
    ``linear`` N(0, 0.02), ``bias`` N(0, 0.02), ``norm`` 1 + N(0, 0.02), ``eye`` identity + N(0, 0.02)
    (a square matrix), ``ids`` an integer table whose rows hold distinct ids below ``arg`` (stored as
    int32; every other kind is a floating-point tensor)."""
    name: str
    shape: tuple[int, ...]
    init: str = "linear"
    optional: bool = False
    arg: int = 0


@dataclass(frozen=True)
class CacheTensor:
    """One paged tensor of a mixer's cache: per token ``heads`` rows of ``width`` elements,
    laid out ``[pages, heads, page_size, width]``."""
    name: str
    heads: int
    width: int


@dataclass(frozen=True)
class PagedCache:
    """What a mixer wants cached per token, in pages: any number of tensors (keys and values, or
    one latent vector, ...).  ``window`` None keeps every token, W keeps the last W (older pages go
    back to the pool) and, with ``keep_first`` k, the first k as well.  ``page_size`` None takes the
    engine's page size; layers whose window, kept tokens and page size agree share a pool of pages and a
    block table."""
    tensors: tuple[CacheTensor, ...]
    window: int | None = None
    page_size: int | None = None
    keep_first: int = 0

    def elements_per_token(self) -> int:
        return sum(t.heads * t.width for t in self.tensors)

    def same_layout(self, other: "PagedCache") -> bool:
        return self.tensors == other.tensors and self.page_size == other.page_size


def PagedKV(num_kv_heads: int, head_dim: int, window: int | None = None, page_size: int | None = None,
            keep_first: int = 0) -> PagedCache:
    """The need of an attention mixer: per token ``num_kv_heads * head_dim`` keys (tensor ``k``)
    and as many values (tensor ``v``)."""
    return PagedCache((CacheTensor("k", int(num_kv_heads), int(head_dim)),
                       CacheTensor("v", int(num_kv_heads), int(head_dim))), window, page_size, int(keep_first))


@dataclass(frozen=True)
class RequestState:
    """A mixer's need for a tensor of fixed size per request (zeroed when a request starts).  A part that
    needs several returns a dict ``name -> RequestState`` from ``state_need()`` and asks for each with
    ``ctx.state(call, name)``."""
    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class PartSpec:
    """Which part to build (a name in the registry of its kind) and its parameters."""
    kind: str
    params: dict[str, Any] = field(default_factory=dict)


class Runtime:
    """Device, activation dtype and the kernel backend, handed to every part."""

    def __init__(self, device, dtype: torch.dtype, ops):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"compute dtype must be float32 or bfloat16, got {dtype}")
        self.device = torch.device(device)
        self.dtype = dtype
        self.ops = ops

    def matrix(self, t: torch.Tensor) -> torch.Tensor:
        """A weight matrix in the activation dtype on the device."""
        return t.to(device=self.device, dtype=self.dtype).contiguous()

    def vector(self, t: torch.Tensor) -> torch.Tensor:
        """Norm weights and biases: always 32-bit (they enter 32-bit arithmetic)."""
        return t.to(device=self.device, dtype=torch.float32).contiguous()

    def table(self, t: torch.Tensor) -> torch.Tensor:
        """An integer table (ids) as int32 on the device."""
        return t.to(device=self.device, dtype=torch.int32).contiguous()


class Part:
    # False for a part whose forward reads device data on the host (a synchronisation): steps of a
    # model that holds one are not captured in CUDA graphs.
    graph_safe = True

    def param_specs(self) -> list[ParamSpec]:
        return []

    def load(self, tensors: dict[str, torch.Tensor], rt: Runtime) -> None:
        """``tensors`` maps this part's relative names to the stored tensors (optional ones
        may be absent)."""


class Norm(Part):
    def forward(self, x: torch.Tensor, rt: Runtime, rows: torch.Tensor | None = None,
                out_dtype: torch.dtype | None = None) -> torch.Tensor:
        """Normalises the 32-bit rows ``x`` (only ``rows`` of them when given); the result has
        ``out_dtype``, the runtime's activation dtype when None."""
        raise NotImplementedError

    def pair_with(self, other: "Norm"):
        """None, or a function ``(x_f32, rt, want_f32) -> (a, b, b32)`` that applies this norm and ``other`` to the
        same rows in one pass: a and b in the activation dtype, b once more in 32-bit when ``want_f32`` (else None).
        A block whose two sublayers read the same rows asks for it."""
        return None

    def fusable_rms(self) -> tuple[torch.Tensor, float] | None:
        """``(weight, eps)`` if this norm is a plain RMS norm that a kernel may apply itself to the
        32-bit residual (the router's kernel does), else None: the caller then asks ``forward`` for a
        32-bit result."""
        return None

    def closing(self) -> "tuple[torch.Tensor, torch.Tensor | None, float] | None":
        """``(weight, bias, eps)`` if a kernel may apply this norm to a sublayer's output itself while it adds it to the
        residual: with a bias the centred norm, with bias None the plain RMS norm.  None: the caller asks ``forward``."""
        rms = self.fusable_rms()
        return None if rms is None else (rms[0], None, rms[1])

    def scale_output(self, factor: torch.Tensor) -> None:
        """Multiplies the norm's output entry by entry by ``factor`` (32-bit, once, after ``load``): a learned scale
        behind a norm joins the norm's own weights."""
        raise NotImplementedError(f"{type(self).__name__} cannot take a factor on its output")


class PositionEncoding(Part):
    """``rotary()`` returns None or ``(inv_freq f32[rotary_dim/2] on the device, rotary_dim)``:
    pair i of each head is rotated by ``position * inv_freq[i]``; dimensions from ``rotary_dim``
    on pass through.  Pair i is dims ``(i, i + rotary_dim/2)``, or ``(2i, 2i + 1)`` when the
    class attribute ``interleaved`` is True.  Sines and cosines are multiplied by ``amplitude``."""

    interleaved = False
    amplitude = 1.0

    def rotary(self, rt: Runtime):
        return None

    def on_embed(self, x: torch.Tensor, positions: torch.Tensor, rt: Runtime) -> None:
        """Hook for encodings that act on the embedded tokens (in place); default: nothing."""

    def added_rows(self):
        """The table of an encoding that does no more than add row ``position`` of it to the embedded token (a kernel may
        then do that itself), else None."""
        return None


class Mixer(Part):
    def cache_need(self) -> PagedCache | None:
        return None

    def state_need(self) -> "RequestState | dict[str, RequestState] | None":
        return None

    def forward(self, h: torch.Tensor, resid: torch.Tensor, ctx: "StepContext", call: int) -> None:
        raise NotImplementedError


class FeedForward(Part):
    # True for a part whose ``forward`` takes ``normed32``: its normalised input once more in 32-bit, when the block
    # has it at hand (it then need not apply ``pre_norm`` again itself)
    takes_normed32 = False

    def forward(self, h: torch.Tensor, resid: torch.Tensor, ctx: "StepContext", pre_norm: "Norm | None" = None) -> None:
        """``pre_norm`` is the norm that produced ``h`` from ``resid``; a part that needs the
        normalised input in 32-bit (a router) may apply it again to the residual itself."""
        raise NotImplementedError


@dataclass
class GroupView:
    """What one cache group contributes to a step: where the new tokens' keys and values go
    and each request's block table."""
    slots: torch.Tensor         # i32 [T]   page * page_size + offset
    block_table: torch.Tensor   # i32 [R, width]
    page_size: int
    window: int                 # 0: none


@dataclass
class StepBatch:
    """Device-side description of one step: a flat array of tokens of several requests."""
    num_tokens: int
    num_requests: int
    tokens: torch.Tensor        # i32 [T]
    positions: torch.Tensor     # i32 [T]  absolute position of each token in its request
    token_req: torch.Tensor     # i32 [T]  row of the request each token belongs to
    cu_q: torch.Tensor          # i32 [R+1] start of each request's tokens
    kv_len: torch.Tensor        # i32 [R]  tokens the request holds after this step
    state_slot: torch.Tensor    # i32 [R]  the request's state slot
    logit_rows: torch.Tensor    # i32 [N]  flat places whose logits are wanted
    groups: list[GroupView]
    max_q_len: int
    max_kv_len: int
    num_single: int = 0         # requests with exactly one token in this step


@dataclass
class PagedView:
    tensors: dict[str, torch.Tensor]   # by CacheTensor.name: [pages, heads, page_size, width]
    group: GroupView
    write: bool                 # False when this call only reads another call's cache

    @property
    def k(self) -> torch.Tensor:
        return self.tensors["k"]

    @property
    def v(self) -> torch.Tensor:
        return self.tensors["v"]


class StepContext:
    """What a mixer or feed-forward may ask for during a step."""

    def __init__(self, rt: Runtime, batch: StepBatch, paged_of_call: Callable[[int], PagedView | None],
                 state_of_call: Callable[..., torch.Tensor | None]):
        self.rt = rt
        self.batch = batch
        self._paged = paged_of_call
        self._state = state_of_call
        self._rounded = None        # (call, rows): what ``leave_rounded`` was given last
        self._zeroed = None         # rows of zeros that a block is done with

    def paged(self, call: int) -> PagedView:
        v = self._paged(call)
        if v is None:
            raise RuntimeError(f"layer call {call} asked for paged keys/values but declared no need for them")
        return v

    def state(self, call: int, name: str = "") -> torch.Tensor:
        """The ``[slots, *shape]`` tensor of a declared per-request state (``name``: its key when the part
        declared several)."""
        s = self._state(call, name) if name else self._state(call)
        if s is None:
            raise RuntimeError(f"layer call {call} asked for per-request state {name!r} but declared no need for it")
        return s

    # ---- rows that blocks with a norm on their sublayers' outputs hand on to each other within a step
    def rounded(self, call: int, resid: torch.Tensor) -> torch.Tensor:
        """The residual in the activation dtype: what the block of the call before left, else a copy made now (in
        32-bit the residual itself)."""
        if self.rt.dtype == torch.float32:
            return resid
        if self._rounded is not None and self._rounded[0] == call - 1:
            return self._rounded[1]
        return self.rt.ops.activation(resid, "copy", self.rt.dtype)

    def leave_rounded(self, call: int, rows: "torch.Tensor | None") -> None:
        """``rows``: the residual after ``call``, rounded (None: whoever changes the residual without rounding it)."""
        self._rounded = None if rows is None else (call, rows)

    def take_zeroed(self, like: torch.Tensor) -> torch.Tensor:
        """32-bit rows of zeros of ``like``'s shape for a sublayer to add into; ``give_zeroed`` takes them back once
        they are zeros again."""
        z, self._zeroed = self._zeroed, None
        return z if z is not None and z.shape == like.shape else torch.zeros_like(like)

    def give_zeroed(self, rows: torch.Tensor) -> None:
        self._zeroed = rows
