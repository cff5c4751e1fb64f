"""Small Gakenex configurations and random weights for the tests.

The weights are drawn so that every mechanism matters to the logits: queries and keys of a size that makes scores
uneven, norm weights away from one, convolutions whose earlier taps weigh as much as the last, the two lambda products
of unlike sizes, gates on both sides of zero, gate and up projections that reach their limits, router scores that are
spread.  Matrices are stored in bfloat16 (so that a bfloat16 engine and the 64-bit plain implementation read the same
numbers).

A, B, C and D differ in every size and option; sizes that a config could make equal by accident (2 dim and vdim, the
windows and kept tokens of two layers, top and 1) are unequal.  A: windows and kept tokens that are no multiple of a
page, a layer without feed-forward, values wider than two keys and narrower.  B: odd sizes, as many key/value heads as
query heads, one key/value head, a window of one token, two taps, five taps.  C: sizes of the tensor-core paths (stored
heads of 128, 64 and 96).  D: no window, a window without kept tokens, more kept tokens than the window holds, no
convolution, a single tap, all experts chosen, no cap on the logits.
"""
from __future__ import annotations

import json
import math
import os

import torch


def attention(heads, kv, dim, vdim, scale, diff, conv=None, window=None, keep=None):
    out = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if conv is not None:
        out["conv"] = conv
    if window is not None:
        out["mask"] = {"size": window} if keep is None else {"size": window, "keep_first": keep}
    return out


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, eps=1e-5, cap=12.0, positions=640):
    out = {"architecture": "Gakenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
           "max_positions": positions}
    if cap:
        out["logit_softcap"] = cap
    return out


CONFIGS = {
    "A": model(131, 96, [
        layer(attention(6, 3, 20, 56, 0.5, 0.25, 4, 19, 21), dense(70, 1.5)),
        layer(attention(4, 1, 28, 24, 0.4, 0.6, 3, 37, 5), moe(9, 2, 30)),
        layer(attention(2, 2, 16, 32, 0.7, 0.1, 2, 19, 21)),
        layer(attention(8, 4, 12, 20, 0.6, 0.45, 4, 50, 33), moe(5, 1, 44))]),
    "B": model(77, 63, [
        layer(attention(5, 5, 7, 9, 0.8, 0.3, 2, 1, 3), dense(33, 0.9)),
        layer(attention(3, 1, 9, 23, 0.5, 0.75, 5, 13, 1), moe(7, 3, 21)),
        layer(attention(2, 1, 5, 3, 1.1, 0.5, 3, 27, 17), dense(18, 4.0))], eps=3e-6, cap=5.0),
    "C": model(264, 192, [
        layer(attention(8, 2, 64, 128, 0.2, 0.35, 4, 100, 70), dense(320, 2.5)),
        layer(attention(6, 3, 32, 64, 0.3, 0.2, 3, 150, 9), moe(12, 2, 96)),
        layer(attention(4, 4, 48, 40, 0.25, 0.55, 2, 65, 130), dense(128, 1.2)),
        layer(attention(16, 1, 56, 72, 0.22, 0.4, 3, 64, 64), moe(8, 1, 64))], eps=1e-6, cap=20.0),
    "D": model(53, 48, [
        layer(attention(4, 2, 12, 20, 0.7, 0.15, 4), moe(3, 3, 22)),
        layer(attention(2, 1, 10, 30, 0.5, 0.8, None, 11), dense(25, 0.7)),
        layer(attention(6, 2, 8, 12, 0.9, 0.33, 1, 6, 40), moe(4, 1, 14)),
        layer(attention(3, 3, 14, 16, 0.6, 0.5, 3, None), dense(31, 3.0))], eps=2e-5, cap=None),
}


def one_layer(lyr, width=64, vocab=53):
    """A model of a single layer (for a mechanism alone)."""
    return model(vocab, width, [lyr])


def make_weights(cfg, seed=0):
    """name -> tensor (bfloat16) for a config dict."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def rnd(*shape, std=1.0, mean=0.0):
        return (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    def lin(o, i, gain=1.0):
        return rnd(o, i, std=gain / math.sqrt(i))

    out["embed"], out["pos"] = rnd(V, W, std=0.8), rnd(cfg["max_positions"], W, std=0.4)
    out["embed.norm"], out["final.norm"] = rnd(W, std=0.25, mean=-0.2), rnd(W, std=0.25, mean=-0.4)
    for i, L in enumerate(cfg["layers"]):
        out[f"l{i}.norm1"] = rnd(W, std=0.25, mean=0.2)
        p, m = f"l{i}.mix.", L["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        rows = {"q": 2 * H * d, "k": 2 * G * d, "v": G * dv}
        for n, r in rows.items():
            out[p + n] = lin(r, W)
            if m.get("conv"):
                out[p + n + ".conv"] = rnd(r, m["conv"], std=0.7)
        for n in "qk":
            out[p + n + ".norm"] = rnd(d, std=0.3, mean=1.6)
        # lambda: exp(about 0.4) - exp(about 0.3) + diff, so that both products and the constant count
        for n, mean in (("lq1", 0.6), ("lk1", 0.65), ("lq2", 0.65), ("lk2", 0.45)):
            out[p + n] = rnd(d, std=0.2, mean=mean) / math.sqrt(d)
        out[p + "g"], out[p + "o"] = lin(H * dv, W, 2.0), lin(W, H * dv, 1.2)
        mlp = L.get("mlp")
        p = f"l{i}.mlp."
        if mlp and mlp["kind"] == "dense":
            out[p + "gate"], out[p + "up"], out[p + "down"] = lin(mlp["ff"], W, 2.0), lin(mlp["ff"], W, 1.5), lin(W, mlp["ff"])
        elif mlp:
            ff = mlp["expert"]["ff"]
            out[p + "router"] = lin(mlp["router"]["experts"], W, 1.5)
            for e in range(mlp["router"]["experts"]):
                out[p + f"e{e}.gate"], out[p + f"e{e}.up"] = lin(ff, W, 2.0), lin(ff, W, 2.0)
                out[p + f"e{e}.down"] = lin(W, ff, 1.5)
    return out


def write_model(cfg, folder, seed=0, tensors=None):
    from dlm_b200.weights.safetensors_io import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    tensors = make_weights(cfg, seed) if tensors is None else tensors
    save_file(tensors, os.path.join(folder, "model.safetensors"))
    return tensors


def tokens(seed, length, vocab):
    g = torch.Generator().manual_seed(17000 + seed)
    return torch.randint(0, vocab, (length,), generator=g).tolist()


def row_error(got, ref):
    """Per row: root mean square of the difference (its mean taken off) over that of the reference."""
    got, ref = got.double(), ref.double()
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    r = ref - ref.mean(-1, keepdim=True)
    return torch.sqrt((d * d).mean(-1)) / torch.sqrt((r * r).mean(-1))


# what a correct engine stays within (rounding of the format; measured values are printed by the tests)
TOL = {"float32": 1e-4, "bfloat16": 3e-2}
# Where the choice of experts hangs on a gap between logits that rounding can close, two correct computations choose
# differently.  Requests are made so that there is none (``clear_requests``); a position that is left over, and those
# behind it (they read its keys), get no limit.
MARGIN = {"float32": 1e-5, "bfloat16": 0.05}


_CLEAR = {}


def clear_requests(oracle, lengths, seed=0):
    """``{"r0": tokens, ...}`` of the given lengths without a close choice of experts: tokens at which the plain model's
    routing is close are drawn anew, from the front, until none is."""
    key = (json.dumps(oracle.cfg), float(oracle.t["embed"].sum()), tuple(lengths), seed)
    if key in _CLEAR:
        return dict(_CLEAR[key])
    g = torch.Generator().manual_seed(23000 + seed)
    V, out = oracle.cfg["vocab"], {}
    for r, n in enumerate(lengths):
        t = torch.randint(0, V, (n,), generator=g)
        for _ in range(150):
            close = oracle.router_margins(t.tolist()) < 1.2 * MARGIN["bfloat16"]
            if not bool(close.any()):
                break
            t[close] = torch.randint(0, V, (int(close.sum()),), generator=g)
        out[f"r{r}"] = t.tolist()
    _CLEAR[key] = out
    return dict(out)


def references(oracle, reqs, dtype):
    """Per request the exact logits and a limit for every position: TOL, or in bfloat16 three times the error that
    rounding alone causes (the plain model with bfloat16 where an engine must round) where that is more.  The error
    rounding causes at a position is taken as the larger of the rounded run's error there and its root mean square over
    the request.  From the first position on whose routing hangs on a close call the limit is infinite."""
    import plain_gakenex as plain
    ref = {rid: oracle.forward(t) for rid, t in reqs.items()}
    lim = {rid: torch.full((len(t),), TOL[dtype], dtype=torch.float64) for rid, t in reqs.items()}
    rounded = plain.PlainGakenex(oracle.cfg, oracle.t, rounded=True)
    for rid, t in reqs.items():
        close = torch.cumsum((oracle.router_margins(t) < MARGIN[dtype]).to(torch.int32), 0) > 0
        if dtype == "bfloat16":
            err = row_error(rounded.forward(t), ref[rid])
            ok = err[~close]
            base = torch.sqrt((ok * ok).mean()) if ok.numel() else torch.tensor(0.0, dtype=torch.float64)
            lim[rid] = torch.maximum(lim[rid], 3.0 * torch.maximum(err, base))
        lim[rid][close] = float("inf")
    return ref, lim


def ratios(got, ref, lim):
    """error / limit for every row of ``{(request, position): logits}`` that has a limit."""
    return [float(row_error(row, ref[rid][p]) / lim[rid][p]) for (rid, p), row in got.items()
            if math.isfinite(float(lim[rid][p]))]
