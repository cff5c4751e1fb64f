"""Small Zepilorn configurations and random weights for the tests.

The weights are drawn so that every mechanism matters to the logits: queries and keys of a size that makes scores
uneven, norm weights away from 1 with biases, layer scales on both sides of 1, gate projections on both sides of zero,
decays between forgetting at once and not at all.  Matrices are stored in bfloat16 (so that a bfloat16 engine and the
64-bit plain implementation read the same numbers).

A, B, C and D differ in every size and option; sizes that a config could make equal by accident (dim and vdim, the
windows of two layers, the rank and a head count) are unequal.  A: all three mixers, a reader of an earlier layer's keys
that looks further back than that layer itself, a layer without feed-forward, windows that are no multiple of a page.
B: sizes that are multiples of neither 4 nor 8, as many key/value heads as query heads, a rotation over the whole head
without scaling, one recurrent head, a window of one token.  C: sizes of the tensor-core paths (128- and 64-wide heads,
a latent of 128).  D: no rotation, no window in one layer, two readers of one layer (one looks less far, one without a
window), a latent wider than a warp's share, decays of exactly 1 and 0.
"""
from __future__ import annotations

import json
import math
import os

import torch


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads, kv, dim, vdim, scale, window=None, base=None, dims=None, scaling=None, kv_from=None):
    out = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        out["mask"] = {"size": window}
    if base is not None:
        out["rot"] = {"base": base, "dims": dims if dims is not None else dim}
        if scaling:
            out["rot"]["scaling"] = scaling
    if kv_from is not None:
        out["kv_from"] = kv_from
    return out


def latent(heads, dim, vdim, rank, scale, window=None):
    out = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale}
    if window is not None:
        out["mask"] = {"size": window}
    return out


def linear(dim, vdim, decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def layer(mixer, ff=None):
    kind = "lightning" if "decay" in mixer else ("latent_attention" if "kv_rank" in mixer else "attention")
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(vocab, width, layers, eps=1e-5):
    return {"architecture": "Zepilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


_ROT_A = dict(base=5000.0, dims=16, scaling=yarn(6.0, 96, 8.0, 0.5))
CONFIGS = {
    "A": model(131, 96, [
        layer(attention(6, 3, 24, 40, 1.3, 19, **_ROT_A), 70),
        layer(linear(10, 14, [0.5, 0.93, 0.995]), 44),
        layer(attention(9, 3, 24, 40, 0.9, 45, kv_from=0, **_ROT_A)),
        layer(latent(5, 20, 12, 28, 0.5, 33), 100),
        layer(attention(3, 3, 24, 40, 1.7, 7, kv_from=0, **_ROT_A), 30)]),
    "B": model(77, 62, [
        layer(latent(3, 7, 9, 22, 0.8, 13), 26),
        layer(attention(5, 5, 10, 6, 1.9, 1, base=300.0), 34),
        layer(linear(9, 5, [0.8]), 50),
        layer(attention(2, 1, 18, 14, 1.1, 27, base=77.0, dims=6), 18)], eps=3e-6),
    "C": model(264, 192, [
        layer(attention(4, 1, 128, 128, 1.2, 150, base=1e6, dims=64, scaling=yarn(4.0, 256, 16.0, 1.0)), 320),
        layer(latent(8, 64, 48, 128, 0.3, 90), 160),
        layer(linear(32, 64, [0.7, 0.98, 0.999, 0.9]), 96),
        layer(attention(8, 2, 64, 96, 1.0, 70, base=1e4, dims=32), 128),
        layer(attention(2, 1, 128, 128, 0.8, 260, base=1e6, dims=64, scaling=yarn(4.0, 256, 16.0, 1.0), kv_from=0), 64)],
        eps=1e-6),
    "D": model(53, 48, [
        layer(attention(4, 2, 12, 20, 1.5, 11), 22),
        layer(attention(2, 2, 12, 20, 1.2, 5, kv_from=0), 30),
        layer(linear(8, 12, [1.0, 0.0, 0.6]), 14),
        layer(attention(6, 2, 12, 20, 0.7, None, kv_from=0)),
        layer(latent(2, 16, 10, 72, 0.6), 26)], eps=2e-5),
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

    def norm(name, size=W):
        out[name], out[name + ".b"] = rnd(size, std=0.2, mean=1.0), rnd(size, std=0.15)

    out["embed"], out["head"] = rnd(V, W, std=0.8), lin(V, W, gain=2.0)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        norm(f"l{i}.norm1")
        out[f"l{i}.ls1"] = rnd(W, std=0.3, mean=0.9)
        p, m = f"l{i}.mix.", L["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        out[p + "o"] = lin(W, H * dv)
        if L["type"] == "attention":
            out[p + "q"] = lin(H * d, W, 1.5)
            if m.get("kv_from") is None:
                out[p + "k"], out[p + "v"] = lin(m["kv_heads"] * d, W, 1.5), lin(m["kv_heads"] * dv, W, 1.2)
        elif L["type"] == "latent_attention":
            r = m["kv_rank"]
            out[p + "q"], out[p + "dkv"], out[p + "dkv.norm"] = lin(H * d, W, 1.5), lin(r, W), rnd(r, std=0.2, mean=1.1)
            out[p + "uk"], out[p + "uv"] = lin(H * d, r, 1.3), lin(H * dv, r, 1.2)
        else:
            out[p + "q"], out[p + "k"], out[p + "v"] = lin(H * d, W, 1.2), lin(H * d, W, 1.2), lin(H * dv, W, 1.5)
            out[p + "g"], out[p + "norm"] = lin(H * dv, W, 2.0), rnd(H * dv, std=0.3, mean=1.1)
        if L.get("mlp"):
            ff = L["mlp"]["ff"]
            norm(f"l{i}.norm2")
            out[f"l{i}.ls2"] = rnd(W, std=0.3, mean=0.8)
            p = f"l{i}.mlp."
            out[p + "gate"], out[p + "up"], out[p + "down"] = lin(ff, W, 1.5), lin(ff, W, 1.2), lin(W, ff)
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
    g = torch.Generator().manual_seed(11000 + seed)
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


def references(oracle, reqs, dtype):
    """Per request the exact logits and a limit for every position: TOL, or in bfloat16 three times the error that
    rounding alone causes (the plain model with bfloat16 where an engine must round) where that is more.  The error
    rounding causes at a position is taken as the larger of the rounded run's error there and its root mean square
    over the request."""
    import plain_zepilorn as plain
    ref = {rid: oracle.forward(t) for rid, t in reqs.items()}
    lim = {rid: torch.full((len(t),), TOL[dtype], dtype=torch.float64) for rid, t in reqs.items()}
    if dtype == "bfloat16":
        rounded = plain.PlainZepilorn(oracle.cfg, oracle.t, rounded=True)
        for rid, t in reqs.items():
            err = row_error(rounded.forward(t), ref[rid])
            err = torch.maximum(err, torch.sqrt((err * err).mean()))
            lim[rid] = torch.maximum(lim[rid], 3.0 * err)
    return ref, lim


def ratios(got, ref, lim):
    """error / limit for every row of ``{(request, position): logits}``."""
    return [float(row_error(row, ref[rid][p]) / lim[rid][p]) for (rid, p), row in got.items()]
