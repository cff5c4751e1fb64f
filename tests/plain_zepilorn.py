"""A plain, slow statement of the Zepilorn design in PyTorch, one function per mechanism.

It shares no code with the package: it reads ``config.json`` as a dict and the
tensors by their stored names, walks the recurrence token by token, and keeps
nothing between calls.  Everything is computed in ``dtype`` (float64 by default)
from the weights as they are stored.  With ``rounded=True`` whatever a 16-bit
engine hands to a matrix product or keeps in its cache is rounded to bfloat16
first.

Notation: ``h`` is a sublayer's input ``[T, width]``; ``p(name)`` gives a tensor of
the current layer's mixer or feed-forward; positions count from 0.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ small pieces
def as_stored(x, rounded):
    return x.to(torch.bfloat16).to(x.dtype) if rounded else x


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def yarn(base, dims, scaling):
    """(frequencies ``f_i``, i < dims / 2, in 64-bit; the factor on sines and cosines).  With ``scaling`` (factor,
    original, fast, slow): the entry whose wave turns t times within ``original`` positions is
    ``dim(t) = dims ln(original / (2 pi t)) / (2 ln base)``; below ``lo = max(floor dim(fast), 0)`` a frequency is
    kept, above ``hi = min(ceil dim(slow), dims - 1)`` it is divided by ``factor``, in between it is blended linearly."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, orig, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))

    def dim(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))

    lo, hi = max(math.floor(dim(fast)), 0), min(math.ceil(dim(slow)), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / factor * ramp + x * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, freqs, dims, amplitude):
    """First ``dims`` entries of the last dimension, entry i with entry i + dims / 2; x: [T, heads, D]."""
    if dims == 0:
        return x
    half = dims // 2
    a = (positions.to(x.dtype)[:, None] * freqs.to(x.dtype)[None, :])[:, None, :]
    c, s = amplitude * torch.cos(a), amplitude * torch.sin(a)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(T, window):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    return see & (i - j < window) if window else see


# ------------------------------------------------------------------------ mixers
def rotated_unit_heads(x, m, eps):
    """Rotation first, then every head divided by its root mean square."""
    rot = m.get("rot")
    if rot and rot.get("dims"):
        f, amp = yarn(rot["base"], rot["dims"], rot.get("scaling"))
        x = rotate_halves(x, torch.arange(x.shape[0]), f, rot["dims"], amp)
    return unit_rms(x, eps)


def attention_keys_values(h, p, m, eps, rounded=False):
    """What a layer with key and value projections keeps per token: rotated unit keys and values."""
    G, T = m["kv_heads"], h.shape[0]
    hh = as_stored(h, rounded)
    k = rotated_unit_heads((hh @ p("k").T).reshape(T, G, m["dim"]), m, eps)
    v = (hh @ p("v").T).reshape(T, G, m["vdim"])
    return as_stored(k, rounded), as_stored(v, rounded)


def sink_softmax(s):
    """exp(s) / (1 + sum exp(s)) over the last dimension (masked scores are -inf)."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def windowed_attention(h, p, m, eps, kv, rounded=False):
    """Grouped-query attention over the last ``window`` tokens with a silent sink; ``kv``: keys and values (this
    layer's own or an earlier layer's)."""
    H, G, T = m["heads"], m["kv_heads"], h.shape[0]
    hh = as_stored(h, rounded)
    q = as_stored(rotated_unit_heads((hh @ p("q").T).reshape(T, H, m["dim"]), m, eps), rounded)
    k, v = (x.repeat_interleave(H // G, dim=1) for x in kv)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    s = s.masked_fill(~visible(T, (m.get("mask") or {}).get("size"))[None], float("-inf"))
    o = torch.einsum("hij,jhv->ihv", sink_softmax(s), v).reshape(T, H * m["vdim"])
    return as_stored(o, rounded) @ p("o").T


def latent_attention(h, p, m, eps, rounded=False):
    """Attention without positions whose keys and values are projections of one normed latent per token."""
    H, d, dv, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    hh = as_stored(h, rounded)
    q = as_stored((hh @ p("q").T).reshape(T, H, d), rounded)
    c = as_stored(unit_rms(hh @ p("dkv").T, eps) * p("dkv.norm"), rounded)
    k = as_stored((c @ p("uk").T).reshape(T, H, d), rounded)
    v = as_stored((c @ p("uv").T).reshape(T, H, dv), rounded)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    s = s.masked_fill(~visible(T, (m.get("mask") or {}).get("size"))[None], float("-inf"))
    o = torch.einsum("hij,jhv->ihv", torch.softmax(s, dim=-1), v).reshape(T, H * dv)
    return as_stored(o, rounded) @ p("o").T


def lightning(h, p, m, eps, rounded=False, state=None):
    """Linear attention with a constant decay per head on silu'd projections; one norm over all heads together and a
    sigmoid gate.  ``state`` continues an earlier call; the new one is returned beside the output."""
    H, d, dv, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    hh = as_stored(h, rounded)
    q, k = (silu(hh @ p(n).T).reshape(T, H, d) for n in "qk")
    v = silu(hh @ p("v").T).reshape(T, H, dv)
    decay = torch.tensor(m["decay"], dtype=h.dtype)[:, None, None]
    S = torch.zeros(H, d, dv, dtype=h.dtype) if state is None else state.clone()
    o = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    y = unit_rms(o.reshape(T, H * dv), eps) * p("norm") * sigmoid(hh @ p("g").T)
    return as_stored(y, rounded) @ p("o").T, S


# ------------------------------------------------------------------ feed-forward
def gated_mlp(h, p, rounded=False):
    hh = as_stored(h, rounded)
    return as_stored(gelu_tanh(hh @ p("gate").T) * (hh @ p("up").T), rounded) @ p("down").T


# ------------------------------------------------------------------------- model
class PlainZepilorn:
    """``tensors``: name -> tensor as stored.  ``forward(tokens)`` gives logits at every position and, with
    ``trace=True``, also the residual after every layer."""

    def __init__(self, config: dict, tensors: dict, dtype=torch.float64, rounded=False):
        self.cfg, self.dtype, self.rounded = config, dtype, rounded
        self.eps = config["norm"]["eps"]
        self.t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}

    def norm(self, name, x):
        return layer_norm(x, self.t[name], self.t[name + ".b"], self.eps)

    def mixer(self, i, x, kept):
        spec = self.cfg["layers"][i]
        m, t, eps, r = spec["mixer"], self.t, self.eps, self.rounded
        p = lambda n: t[f"l{i}.mix.{n}"]
        if spec["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = attention_keys_values(x, p, m, eps, r)
            return windowed_attention(x, p, m, eps, kept[i if src is None else src], r)
        if spec["type"] == "latent_attention":
            return latent_attention(x, p, m, eps, r)
        assert spec["type"] == "lightning"
        return lightning(x, p, m, eps, r)[0]

    def layer(self, i, x, kept):
        t = self.t
        x = x + self.norm(f"l{i}.norm1", self.mixer(i, x, kept)) * t[f"l{i}.ls1"]
        mlp = self.cfg["layers"][i].get("mlp")
        if mlp is not None:
            assert mlp["kind"] == "dense"
            x = x + self.norm(f"l{i}.norm2", gated_mlp(x, lambda n: t[f"l{i}.mlp.{n}"], self.rounded)) * t[f"l{i}.ls2"]
        return x

    def forward(self, tokens, trace=False):
        x = self.t["embed"][torch.as_tensor(tokens, dtype=torch.long)].clone()
        after, kept = [], {}
        for i in range(len(self.cfg["layers"])):
            x = self.layer(i, x, kept)
            after.append(x)
        logits = as_stored(self.norm("final.norm", x), self.rounded) @ self.t["head"].T
        return (logits, torch.stack(after)) if trace else logits
