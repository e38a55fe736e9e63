"""A plain, slow Nufatar in float64: one function per mechanism, whole sequences only, no cache and no batching.

It shares no code with the package: it reads the checkpoint's own tensor names (`embed`, `loop.step`, `l<i>.norm1`,
`l<i>.mix.left.q`, ...) from a dict of tensors and the checkpoint's own `config.json` dict.  The package's tests compare every path
of the framework (packed prefill, token-by-token decoding through the state manager, batches, generation) with it.

Notation: x [T, W] is one sequence's residual stream, positions 0 .. T - 1.
"""

from __future__ import annotations

import math
from typing import Dict, List

import torch

F64 = torch.float64


def rms_divide(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    return rms_divide(x, eps) * (1.0 + w)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


# ------------------------------------------------------------------------------------------------ attention


def distance_bucket(n: int, rows: int, bias_max: float) -> int:
    """Row of the bias table for distance n: exact below rows / 2, then logarithmic up to bias_max, the last row beyond."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (rows - half)))


def frequencies(rot: dict):
    """(frequencies [dims / 2], factor on cos and sin)."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return torch.tensor(f, dtype=F64), 1.0
    at = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_half(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, H, d]: the pairs (i, i + dims / 2) of the first `dims` dimensions turn by position * f_i, scaled by the factor."""
    f, m = frequencies(rot)
    n = rot["dims"] // 2
    ang = torch.arange(x.shape[0], dtype=F64).unsqueeze(1) * f
    cs, sn = (torch.cos(ang) * m).unsqueeze(1), (torch.sin(ang) * m).unsqueeze(1)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * cs - v * sn, v * cs + u * sn, x[..., 2 * n:]], -1)


def attend(q, k, v, scale, window=None, bias=None, sink=None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv].  bias [T, H]: what is added to the scaled score at every distance; sink [H]."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = torch.arange(T).unsqueeze(1), torch.arange(T).unsqueeze(0)
    ok = j <= i
    if window is not None:
        ok = ok & (i - j < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[(i - j).clamp(min=0), h]
        s = s.masked_fill(~ok, -math.inf)
        mx = s.max(-1, keepdim=True).values
        if sink is not None:
            mx = torch.maximum(mx, sink[h])
        e = torch.exp(s - mx)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - mx)
        out[:, h] = (e / den) @ v[:, g]
    return out


def biased_attention(w, m: dict, h: torch.Tensor) -> torch.Tensor:
    """Left side of `parallel`: keys are the values, learned distance bias, window, sink.  w: name -> float64 tensor."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    rel = w["rel"]
    q, k = (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, G, d)
    bias = rel[torch.tensor([distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)])]
    mask = m.get("mask")
    o = attend(q, k, k, m["scale"], mask["size"] if mask else None, bias, w["sink"])
    return o.reshape(T, -1) @ w["o"].T


def rotated_attention(w, m: dict, h: torch.Tensor) -> torch.Tensor:
    """Left side of `parallel_2`: rotated queries and keys, every earlier token visible, ordinary softmax."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, G, d)
    if m.get("rot"):
        q, k = rotate_half(q, m["rot"]), rotate_half(k, m["rot"])
    mask = m.get("mask")
    return attend(q, k, (h @ w["v"].T).view(T, G, dv), m["scale"], mask["size"] if mask else None).reshape(T, -1) @ w["o"].T


# ------------------------------------------------------------------------------------------------ gated delta rule


def short_conv_silu(x: torch.Tensor, cw: torch.Tensor) -> torch.Tensor:
    """x [T, C], cw [C, taps] (the last tap meets the current token); inputs before the first token are zero; then silu."""
    T, taps = x.shape[0], cw.shape[1]
    y = torch.zeros_like(x)
    for back in range(min(taps, T)):
        y[back:] += x[:T - back] * cw[:, taps - 1 - back]
    return silu(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_core(q, k, v, beta, decay) -> torch.Tensor:
    """q, k [T, G, d], v [T, H, dv], beta [T, H], decay [T, H, d] (one factor per row of S).  S starts at zero; returns o [T, H, dv]."""
    T, H, dv = v.shape
    q, k = (x.repeat_interleave(H // x.shape[1], 1) for x in (q, k))      # head h reads q / k head floor(h / (H / G))
    o = torch.zeros(T, H, dv, dtype=F64)
    S = torch.zeros(H, q.shape[2], dv, dtype=F64)
    for t in range(T):
        S = decay[t].unsqueeze(-1) * S
        u = beta[t].unsqueeze(-1) * (v[t] - (k[t].unsqueeze(1) @ S).squeeze(1))
        S = S + k[t].unsqueeze(-1) * u.unsqueeze(1)
        o[t] = (q[t].unsqueeze(1) @ S).squeeze(1)
    return o


def delta_rule(w, m: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Right side of both mixers.  A decay per key channel and a sigmoid gate, both through two factors (`a1`, `a2`, `g1`, `g2`), or one
    decay per head and a silu gate (`a`, `g`)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(short_conv_silu(h @ w["q"].T, w["q.conv"]).view(T, G, d)) * d ** -0.5
    k = unit(short_conv_silu(h @ w["k"].T, w["k.conv"]).view(T, G, d))
    v = short_conv_silu(h @ w["v"].T, w["v.conv"]).view(T, H, dv)
    beta = sigmoid(h @ w["b"].T)
    if "a1" in w:
        z = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
        z = z.view(T, H, d)
        gate = sigmoid((h @ w["g1"].T) @ w["g2"].T)
    else:
        z = (h @ w["a"].T + w["dt_bias"]).view(T, H, 1).expand(T, H, d)
        gate = silu(h @ w["g"].T)
    softplus = torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)
    decay = torch.exp(-torch.exp(w["A_log"]).view(1, H, 1) * softplus)
    o = rms_divide(delta_core(q, k, v, beta, decay), eps) * w["norm"]
    return (o.reshape(T, H * dv) * gate) @ w["o"].T


# ------------------------------------------------------------------------------------------------ blocks


def side(sd, pre: str) -> Dict[str, torch.Tensor]:
    return {k[len(pre):]: t.to(F64) for k, t in sd.items() if k.startswith(pre)}


def mixer(sd, lay: dict, pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    m = lay["mixer"]
    wl, wr = side(sd, pre + "left."), side(sd, pre + "right.")
    right = delta_rule(wr, m["right"], h, eps)
    if lay["type"] == "parallel":
        left = biased_attention(wl, m["left"], h)
        return 0.5 * (rms_divide(left, eps) * wl["out"] + rms_divide(right, eps) * wr["out"])
    assert lay["type"] == "parallel_2"
    return m["left_scale"] * rotated_attention(wl, m["left"], h) + m["right_scale"] * right


def feed_forward(sd, pre: str, h: torch.Tensor) -> torch.Tensor:
    w = side(sd, pre)
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def layer(sd, cfg: dict, i: int, x: torch.Tensor) -> torch.Tensor:
    lay, eps = cfg["layers"][i], cfg["norm"]["eps"]
    h = one_plus_norm(x, sd[f"l{i}.norm1"].to(F64), eps)
    y = mixer(sd, lay, f"l{i}.mix.", h, eps)
    if lay.get("mlp") is not None:
        y = y + feed_forward(sd, f"l{i}.mlp.", h)
    return x + y


def run_order(cfg: dict) -> List[tuple]:
    """(layer, number of the pass that starts right before it or None) for every layer run, in execution order."""
    L, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(L)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, L)]


def forward(sd: Dict[str, torch.Tensor], cfg: dict, tokens: List[int], want_layers: bool = False):
    """Logits [T, vocab] of one sequence (and, if asked, the residual stream after every layer run [runs, T, W])."""
    emb = sd["embed"].to(F64)
    x, trace = emb[torch.tensor(tokens, dtype=torch.long)], []
    for i, t in run_order(cfg):
        if t is not None:
            x = x + sd["loop.step"].to(F64)[t]
        x = layer(sd, cfg, i, x)
        trace.append(x)
    logits = one_plus_norm(x, sd["final.norm"].to(F64), cfg["norm"]["eps"]) @ emb.T
    return (logits, torch.stack(trace)) if want_layers else logits


def greedy(sd, cfg, prompt: List[int], n_new: int) -> List[int]:
    toks, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(forward(sd, cfg, toks)[-1].argmax())
        out.append(nxt)
        toks.append(nxt)
    return out


# ---------------------------------------------------------------------------------------------- random checkpoints for tests


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Shapes of every tensor.  The inner ranks of `parallel`'s right side and the rows of its bias table are not part of a checkpoint's
    config; a test's config names them `decay_rank`, `gate_rank` and `bias_rows`."""
    W = cfg["width"]
    s = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    if cfg.get("loop"):
        s["loop.step"] = (cfg["loop"]["times"], W)
    for i, lay in enumerate(cfg["layers"]):
        l, r, p = lay["mixer"]["left"], lay["mixer"]["right"], f"l{i}."
        s[p + "norm1"] = (W,)
        q = p + "mix.left."
        s.update({q + "q": (l["heads"] * l["dim"], W), q + "k": (l["kv_heads"] * l["dim"], W), q + "o": (W, l["heads"] * l["vdim"])})
        if lay["type"] == "parallel":
            s.update({q + "rel": (l["bias_rows"], l["heads"]), q + "sink": (l["heads"],), q + "out": (W,)})
        else:
            s[q + "v"] = (l["kv_heads"] * l["vdim"], W)
        q = p + "mix.right."
        H, G, d, dv, t = r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]
        s.update({q + "q": (G * d, W), q + "q.conv": (G * d, t), q + "k": (G * d, W), q + "k.conv": (G * d, t), q + "v": (H * dv, W),
                  q + "v.conv": (H * dv, t), q + "b": (H, W), q + "A_log": (H,), q + "norm": (dv,), q + "o": (W, H * dv)})
        if lay["type"] == "parallel":
            ra, rg = r["decay_rank"], r["gate_rank"]
            s.update({q + "a1": (ra, W), q + "a2": (H * d, ra), q + "dt_bias": (H * d,), q + "g1": (rg, W), q + "g2": (H * dv, rg), q + "out": (W,)})
        else:
            s.update({q + "a": (H, W), q + "dt_bias": (H,), q + "g": (H * dv, W)})
        if lay.get("mlp") is not None:
            F = lay["mlp"]["ff"]
            s.update({p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return s


def random_checkpoint(cfg: dict, seed: int = 0, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights whose scales keep every mechanism alive: activations of order one, decays spread over (0, 1), sinks and bias rows
    that differ."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1",) or name == "final.norm":
            t = 0.2 * torch.randn(shape, generator=g)
        elif last in ("norm", "out"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif last in ("rel", "sink"):
            t = torch.randn(shape, generator=g)
        elif last == "A_log":
            t = torch.log(0.2 + 2.0 * torch.rand(shape, generator=g))
        elif last == "dt_bias":
            t = torch.randn(shape, generator=g) - 1.5
        elif last == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        elif name == "loop.step":
            t = 0.7 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * (1.5 / math.sqrt(shape[-1]))
        sd[name] = t.to(dtype)
    return sd
