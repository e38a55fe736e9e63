"""A plain, slow statement of the Tokatar design in PyTorch (float64 by default), one function per mechanism.  It shares no code
with the framework: the tests compare the framework's kernels, caches and schedulers against it.

Inputs are the checkpoint's own names (`embed`, `l<i>.norm1`, `l<i>.mix.q`, ...) and the `config.json` dict.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def frequencies(rot: dict, n: int, scaled: bool = True) -> List[float]:
    """base^(-2i / n) for i < n / 2; with `rot.scaling` the long wavelengths are stretched by `factor`, the short ones kept and
    those between blended linearly in original / wavelength."""
    out = []
    for i in range(n // 2):
        f = rot["base"] ** (-2.0 * i / n)
        sc = rot.get("scaling") if scaled else None
        if sc:
            wavelength = 2.0 * math.pi / f
            if wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wavelength >= sc["original"] / sc["high"]:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, pos, freq: List[float], interleaved: bool):
    """x [T, heads, d]: the first 2 len(freq) dimensions of every head turn by pos * freq; pairs (2i, 2i + 1) or (i, i + n / 2)."""
    n = 2 * len(freq)
    ang = pos.to(x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    first, second = (slice(0, n, 2), slice(1, n, 2)) if interleaved else (slice(0, n // 2), slice(n // 2, n))
    u, v = x[..., first], x[..., second]
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


def attend(q, k, v, first_pos: int, scale: float, chunk: Optional[int] = None, softcap: Optional[float] = None, plus_one: bool = False):
    """q [T, H, d] at positions first_pos .., k [N, G, d] / v [N, G, dv] at positions 0 ..: every query sees j <= i of its own chunk."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    group = torch.arange(H) // (H // G)
    for t in range(T):
        i = first_pos + t
        lo = 0 if chunk is None else (i // chunk) * chunk
        s = torch.einsum("nhd,hd->hn", k[lo:i + 1][:, group], q[t]) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        mx = s.max(1, keepdim=True).values
        if plus_one:
            mx = mx.clamp(min=0.0)
        e = torch.exp(s - mx)
        den = e.sum(1, keepdim=True) + (torch.exp(-mx) if plus_one else 0.0)
        out[t] = torch.einsum("hn,nhd->hd", e / den, v[lo:i + 1][:, group])
    return out


def append(st: dict, name: str, x):
    """The sequence's rows so far with the new ones behind them."""
    st[name] = torch.cat([st[name], x], 0) if name in st else x
    return st[name]


def attention(h, w, m: dict, pos, st: dict):
    """Half-layout rotation (rescaled frequencies), soft-capped scores, chunked, element-wise output gate."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    f = frequencies(m["rot"], m["rot"]["dims"])
    q = rotate((h @ w["q"].T).view(T, H, d), pos, f, False)
    k = append(st, "k", rotate((h @ w["k"].T).view(T, G, d), pos, f, False))
    v = append(st, "v", (h @ w["v"].T).view(T, G, dv))
    o = attend(q, k, v, k.shape[0] - T, m["scale"], (m.get("mask") or {}).get("size"), softcap=m["softcap"])
    return (o.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def attention_2(h, w, m: dict, pos, st: dict, eps: float):
    """Biases, one RMS norm over all query rows and one over all key rows, interleaved rotation of queries, keys and values, one in
    the softmax denominator, chunked; the output turned back by its own position, then gated."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    f = frequencies(m["rot"], m["rot"]["dims"])
    fv = frequencies(m["rot"], dv, scaled=False)
    q = unit_rms(h @ w["q"].T + w["q.b"], eps) * w["q.norm"]
    k = unit_rms(h @ w["k"].T + w["k.b"], eps) * w["k.norm"]
    v = h @ w["v"].T + w["v.b"]
    q = rotate(q.view(T, H, d), pos, f, True)
    k = append(st, "k", rotate(k.view(T, G, d), pos, f, True))
    v = append(st, "v", rotate(v.view(T, G, dv), pos, fv, True))
    o = attend(q, k, v, k.shape[0] - T, m["scale"], (m.get("mask") or {}).get("size"), plus_one=True)
    o = rotate(o, -pos, fv, True)
    return (o.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def latent_attention(h, w, m: dict, pos, st: dict, eps: float):
    """Keys and values up-projected from a normalised latent, one rotated key part (half layout) for all heads; one gate per head."""
    T, H, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    f = frequencies(m["rot"], r)
    q = (h @ w["q"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], pos, f, False)], -1)
    down = h @ w["dkv"].T
    c = append(st, "c", unit_rms(down[:, :rank], eps) * w["dkv.norm"])
    kr = append(st, "kr", rotate(down[:, None, rank:], pos, f, False))
    N = c.shape[0]
    k = torch.cat([(c @ w["uk"].T).view(N, H, d), kr.expand(N, H, r)], -1)
    v = (c @ w["uv"].T).view(N, H, dv)
    o = attend(q, k, v, N - T, m["scale"])
    return (o * torch.sigmoid(h @ w["g"].T)[..., None]).reshape(T, H * dv) @ w["o"].T


def feed_forward(h, w):
    return torch.relu(h @ w["up"].T) ** 2 @ w["down"].T


def branch(x, sub, w, n: str, eps: float):
    """x + ls * rms(sigmoid(W h + b) * sub(h)) * g_b with h = rms(x) * g; the two norms have one factor each."""
    h = unit_rms(x, eps) * w["norm" + n]
    y = sub(h) * torch.sigmoid(h @ w["rg" + n].T + w[f"rg{n}.b"])
    return x + unit_rms(y, eps) * w[f"norm{n}b"] * w["ls" + n]


def sub_dict(sd: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in sd.items() if k.startswith(prefix)}


class Sequence:
    """One sequence's caches, per layer."""

    def __init__(self):
        self.n = 0
        self.layers: Dict[int, dict] = {}


def forward(cfg: dict, sd: Dict[str, torch.Tensor], tokens: List[int], seq: Optional[Sequence] = None, dtype=torch.float64,
            layers_out: Optional[list] = None):
    """Logits [len(tokens), vocab] of `tokens` appended to `seq` (a fresh sequence when None)."""
    sd = {k: v.to(dtype) for k, v in sd.items()}
    seq = seq if seq is not None else Sequence()
    eps = cfg["norm"]["eps"]
    T = len(tokens)
    pos = torch.arange(seq.n, seq.n + T)
    x = sd["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, lay in enumerate(cfg["layers"]):
        w, m = sub_dict(sd, f"l{i}."), lay["mixer"]
        mw, st = sub_dict(w, "mix."), seq.layers.setdefault(i, {})
        mixer = {"attention": lambda h: attention(h, mw, m, pos, st), "attention_2": lambda h: attention_2(h, mw, m, pos, st, eps),
                 "latent_attention": lambda h: latent_attention(h, mw, m, pos, st, eps)}[lay["type"]]
        x = branch(x, mixer, w, "1", eps)
        if lay.get("mlp") is not None:
            x = branch(x, lambda h: feed_forward(h, sub_dict(w, "mlp.")), w, "2", eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    seq.n += T
    return (unit_rms(x, eps) * sd["final.norm"]) @ sd["head"].T


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "head": (V, W), "final.norm": ()}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        mix = {"o": (W, H * dv)}
        if lay["type"] == "latent_attention":
            r, rank = m["rot_dim"], m["kv_rank"]
            mix.update({"q": (H * (d + r), W), "dkv": (rank + r, W), "dkv.norm": (rank,), "uk": (H * d, rank), "uv": (H * dv, rank), "g": (H, W)})
        else:
            G = m["kv_heads"]
            mix.update({"q": (H * d, W), "k": (G * d, W), "v": (G * dv, W), "g": (H * dv, W)})
            if lay["type"] == "attention_2":
                mix.update({"q.b": (H * d,), "k.b": (G * d,), "v.b": (G * dv,), "q.norm": (H * d,), "k.norm": (G * d,)})
        out.update({p + "mix." + k: s for k, s in mix.items()})
        subs = ["1"]
        if lay.get("mlp") is not None:
            F = lay["mlp"]["ff"]
            out.update({p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
            subs.append("2")
        for n in subs:
            out.update({p + "norm" + n: (), p + f"norm{n}b": (), p + "ls" + n: (W,), p + "rg" + n: (W, W), p + f"rg{n}.b": (W,)})
    return out


def random_checkpoint(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Random weights, every value exactly representable in bfloat16 (so that both serving types read the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith(".b"):
            t = 0.5 * torch.randn(shape, generator=g)
        elif len(shape) < 2:                                  # norm factors and weights, layer scales: around 1, never near 0
            t = 1.0 + 0.2 * torch.randn(shape, generator=g).clamp(-3, 3)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * (1.3 / math.sqrt(shape[-1]))
        sd[name] = t.bfloat16().float()
    return sd


def greedy(cfg: dict, sd: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    seq, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(forward(cfg, sd, seq)[-1].argmax())
        out.append(nxt)
        seq.append(nxt)
    return out
