"""A plain, slow statement of the Gakenex design in PyTorch, one function per mechanism.

It shares no code with the package: it reads ``config.json`` as a dict and the
tensors by their stored names, and keeps nothing between calls.  Everything is
computed in ``dtype`` (float64 by default) from the weights as they are stored.
With ``rounded=True`` whatever a 16-bit engine hands to a matrix product or keeps
in its cache is rounded to bfloat16 first.

Notation: ``h`` is a sublayer's input ``[T, width]``; ``p(name)`` gives a tensor of
the current layer's mixer or feed-forward; positions count from 0.
"""
from __future__ import annotations

import torch


# ------------------------------------------------------------------ small pieces
def as_stored(x, rounded):
    return x.to(torch.bfloat16).to(x.dtype) if rounded else x


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def model_norm(x, w, eps):
    """The norm around every layer: its weight is stored as the distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def short_conv(u, w):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) per channel, zeros before the start; ``u`` [T, C], ``w`` [C, taps]."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))


def visible(T, mask):
    """[i, j]: j is not later than i, and lies within the last ``size`` tokens or among the first ``keep_first``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if not mask:
        return see
    return see & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


# ------------------------------------------------------------------------ mixer
def mixing_factor(p, diff):
    """How much of the second map is taken off: exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
    return float(torch.exp((p("lq1") * p("lk1")).sum()) - torch.exp((p("lq2") * p("lk2")).sum()) + diff)


def differential_maps(h, p, m, eps, rounded=False):
    """The two maps' outputs ``[T, H, 2, vdim]``: each an ordinary softmax attention over the same values."""
    H, G, d, dv, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (h @ p(n).T for n in "qkv")
    if m.get("conv"):
        q, k, v = (short_conv(x, p(n + ".conv")) for x, n in ((q, "q"), (k, "k"), (v, "v")))
    q = as_stored(unit_rms(q.reshape(T, H, 2, d), eps) * p("q.norm"), rounded)
    k = as_stored(unit_rms(k.reshape(T, G, 2, d), eps) * p("k.norm"), rounded)
    v = as_stored(v.reshape(T, G, dv), rounded)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihcd,jhcd->hcij", q, k) * m["scale"]
    s = s.masked_fill(~visible(T, m.get("mask"))[None, None], float("-inf"))
    return torch.einsum("hcij,jhv->ihcv", torch.softmax(s, dim=-1), v)


def differential_attention(h, p, m, eps, rounded=False):
    hh = as_stored(h, rounded)
    T = h.shape[0]
    a = as_stored(differential_maps(hh, p, m, eps, rounded), rounded)
    o = a[:, :, 0] - mixing_factor(p, m["diff"]) * a[:, :, 1]
    o = (unit_rms(o, eps) * (1.0 - m["diff"])).reshape(T, -1)
    return as_stored(o * sigmoid(hh @ p("g").T), rounded) @ p("o").T


# ------------------------------------------------------------------ feed-forward
def clamped_mlp(h, p, limit, rounded=False):
    hh = as_stored(h, rounded)
    g = torch.clamp(hh @ p("gate").T, max=limit)
    u = torch.clamp(hh @ p("up").T, min=-limit, max=limit)
    return as_stored(g * sigmoid(1.702 * g) * (u + 1.0), rounded) @ p("down").T


def routing(h, w_router, top):
    """(experts ``[T, top]``, their scores): the largest sigmoid scores, used as they are."""
    s = sigmoid(h @ w_router.T)
    ids = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return ids, torch.gather(s, 1, ids)


def expert(x, p, e, rounded=False):
    g, u = x @ p(f"e{e}.gate").T, x @ p(f"e{e}.up").T
    return as_stored(g * sigmoid(g) * u, rounded) @ p(f"e{e}.down").T


def weighted_input_experts(h, p, top, rounded=False):
    """Each chosen expert sees the token's row times its score; the outputs are added as they are."""
    ids, s = routing(h, p("router"), top)
    hh = as_stored(h, rounded)
    out = torch.zeros_like(h)
    for e in range(p("router").shape[0]):
        for j in range(top):
            rows = (ids[:, j] == e).nonzero().flatten()
            if rows.numel():
                out[rows] += expert(as_stored(s[rows, j:j + 1] * hh[rows], rounded), p, e, rounded)
    return out


# ------------------------------------------------------------------------- model
class PlainGakenex:
    """``tensors``: name -> tensor as stored.  ``forward(tokens)`` gives logits at every position and, with
    ``trace=True``, also the residual after every layer."""

    def __init__(self, config: dict, tensors: dict, dtype=torch.float64, rounded=False):
        self.cfg, self.dtype, self.rounded = config, dtype, rounded
        self.eps = config["norm"]["eps"]
        self.t = {k: v.to(dtype) for k, v in tensors.items()}

    def sublayers(self, i, x):
        """(the normed input, the mixer's output, the feed-forward's output or zeros) of layer i."""
        spec, t, r = self.cfg["layers"][i], self.t, self.rounded
        assert spec["type"] == "attention"
        h = model_norm(x, t[f"l{i}.norm1"], self.eps)
        a = differential_attention(h, lambda n: t[f"l{i}.mix.{n}"], spec["mixer"], self.eps, r)
        mlp, p = spec.get("mlp"), (lambda n: t[f"l{i}.mlp.{n}"])
        if mlp is None:
            return h, a, torch.zeros_like(x)
        if mlp["kind"] == "dense":
            return h, a, clamped_mlp(h, p, mlp["limit"], r)
        assert mlp["kind"] == "moe"
        return h, a, weighted_input_experts(h, p, mlp["router"]["top"], r)

    def router_margins(self, tokens):
        """Per position the smallest gap, over all layers with a router, between the last chosen logit and the next."""
        x = self.embedded(tokens)
        gap = torch.full((len(tokens),), float("inf"), dtype=self.dtype)
        for i, spec in enumerate(self.cfg["layers"]):
            h, a, f = self.sublayers(i, x)
            mlp = spec.get("mlp")
            if mlp and mlp["kind"] == "moe" and mlp["router"]["top"] < mlp["router"]["experts"]:
                top = mlp["router"]["top"]
                z = torch.sort(h @ self.t[f"l{i}.mlp.router"].T, dim=-1, descending=True).values
                gap = torch.minimum(gap, z[:, top - 1] - z[:, top])
            x = x + (a + f)
        return gap

    def embedded(self, tokens):
        x = self.t["embed"][torch.as_tensor(tokens, dtype=torch.long)] + self.t["pos"][:len(tokens)]
        return model_norm(x, self.t["embed.norm"], self.eps)

    def forward(self, tokens, trace=False):
        x = self.embedded(tokens)
        after = []
        for i in range(len(self.cfg["layers"])):
            _, a, f = self.sublayers(i, x)
            x = x + (a + f)
            after.append(x)
        logits = as_stored(model_norm(x, self.t["final.norm"], self.eps), self.rounded) @ self.t["embed"].T
        cap = self.cfg.get("logit_softcap")
        if cap:
            logits = cap * torch.tanh(logits / cap)
        return (logits, torch.stack(after)) if trace else logits
