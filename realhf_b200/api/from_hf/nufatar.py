"""Nufatar checkpoints <-> ReaLModel.

A Nufatar checkpoint is `config.json` + `model.safetensors`.  The config lists the layers one by one (`layers[i]` = mixer type
`parallel` or `parallel_2`, the sizes of its two sides, a feed-forward or null) and a `loop`: a range of layers that runs several times
with the same weights, each pass with its own cache / state, a learned vector added to the stream before every pass.  The model is a
heterogeneous stack (`ReaLModelConfig.blocks`) of mechanisms the config classes offer to any family:

  * `parallel_ff`: one RMSNorm per block (weights stored around zero, `layer_norm_type="gemma"`), mixer and feed-forward read the same
    normalised input and their sum joins an fp32 residual stream; tied embedding;
  * mixer `parallel` of the framework with a delta rule on the right side, for both types.  `parallel`: keys that are also the values, a
    learned distance bias, a sliding window and a sink beside a delta rule with one decay per key channel and a sigmoid gate, both
    through two-factor projections; each side RMS-normalised over the model width (`branch_norm`), half of each.  `parallel_2`:
    half-layout rotation with YaRN scaling beside a delta rule with one decay per head and a SiLU gate; the sides weighed by constants;
  * `BlockMLPConfig(kind="glu")`, `LoopConfig(inject_mode="step")`.

There is no `transformers` class for it: the config is read as a plain dict.  The unit norms' epsilon (1e-6) and the halves of `parallel`
are fixed by the design.  Three sizes are in no config: the rows of the bias table and the inner ranks of the two-factor projections;
`config_from_shapes` takes them from the checkpoint's tensors and enters them as `bias_rows`, `decay_rank` and `gate_rank`.

Checkpoint names -> framework names (layer i of the checkpoint is block i + 1 here):
  embed / final.norm                         0.wte.weight / {L}.ln_f.weight
  loop.step                                  {loop.start+1}.loop_step.weight
  l<i>.norm1                                 attn.ln.weight
  mix.left.q, k, (v), mix.right.q, k, v, ..  attn.in.weight (sections: `sharding.wattn_sections`, then `sharding.delta_sections`)
  mix.left.rel / sink / o / out              attn.rel.weight / attn.sink.weight / attn.o.weight / attn.out_l.weight
  mix.right.q.conv, k.conv, v.conv           attn.conv.weight ([q | k | v] channels x taps)
  mix.right.a2, g2                           attn.low.weight (block-diagonal)
  mix.right.A_log / dt_bias / norm / o / out attn.A_log.weight / dt_bias / o_norm / o2 / out_r
  mlp.gate, up / down                        mlp.gate_up.weight / mlp.down.weight
"""

from __future__ import annotations

import copy
from typing import Dict, List, Tuple

import torch

from realhf_b200.api.model import (BlockConfig, BlockMLPConfig, DeltaRuleConfig, LoopConfig, ReaLModelConfig, RotaryConfig,
                                   WindowAttentionConfig, register_hf_family)

UNIT_EPS = 1e-6                 # inside the root of the delta rule's q / k unit norms
HALVES = (0.5, 0.5)             # `parallel`: the mean of its two normalised sides


def config_from_shapes(d: dict, shapes: Dict[str, Tuple[int, ...]]) -> dict:
    """The config with the sizes that only the tensors carry (sizes already present stay)."""
    d = copy.deepcopy(d)
    for i, lay in enumerate(d["layers"]):
        if lay["type"] != "parallel":
            continue
        pre = f"l{i}.mix."
        for side, key, name in (("left", "bias_rows", "left.rel"), ("right", "decay_rank", "right.a1"), ("right", "gate_rank", "right.g1")):
            if pre + name in shapes:
                lay["mixer"][side].setdefault(key, int(shapes[pre + name][0]))
    return d


def _rotary(rot):
    if not rot:
        return None
    sc = rot.get("scaling")
    kw = dict(factor=float(sc["factor"]), original=sc["original"], fast=float(sc["fast"]), slow=float(sc["slow"]), scaling="yarn") if sc else {}
    return RotaryConfig(dims=int(rot["dims"]), base=float(rot["base"]), interleaved=False, **kw)


def _block(i: int, lay: dict) -> BlockConfig:
    m, f = lay["mixer"], lay.get("mlp")
    if f is not None and f.get("kind", "dense") != "dense":
        raise ValueError(f"Nufatar layer {i}: unknown feed-forward kind `{f['kind']}`")
    if lay["type"] not in ("parallel", "parallel_2"):
        raise ValueError(f"Nufatar layer {i}: unknown mixer type `{lay['type']}`")
    first = lay["type"] == "parallel"
    l, r = m["left"], m["right"]
    mask = l.get("mask")
    if first:
        extra = dict(kv_shared=True, sink=True, bias_rows=int(l["bias_rows"]), bias_max=float(l["bias_max"]))
        low = dict(decay_rank=int(r["decay_rank"]), gate_rank=int(r["gate_rank"]), gate="sigmoid")
    else:
        extra, low = dict(sink=False, rotary=_rotary(l.get("rot"))), dict(gate="silu")
    w = WindowAttentionConfig(n_heads=int(l["heads"]), n_kv_heads=int(l["kv_heads"]), qk_dim=int(l["dim"]), v_dim=int(l["vdim"]), scale=float(l["scale"]),
                              window=int(mask["size"]) if mask else None, keep_first=0, qkv_bias=False, value_norm=False, head_temp=False,
                              slope_base=None, out_gate=False, **extra)
    dl = DeltaRuleConfig(n_heads=int(r["heads"]), n_kv_heads=int(r["kv_heads"]), qk_dim=int(r["dim"]), v_dim=int(r["vdim"]), conv_taps=int(r["conv"]),
                         unit_eps=UNIT_EPS, **low)
    scales = HALVES if first else (float(m["left_scale"]), float(m["right_scale"]))
    return BlockConfig(mixer="parallel", wattn=w, delta=dl, mlp=BlockMLPConfig(kind="glu", ff=int(f["ff"]), act="silu") if f is not None else None,
                       branch_scales=scales, branch_norm=first)


def config_from_dict(d: dict, is_critic: bool = False) -> ReaLModelConfig:
    blocks = [_block(i, lay) for i, lay in enumerate(d["layers"])]
    lp = d.get("loop")
    loop = LoopConfig(start=int(lp["start"]), stop=int(lp["stop"]), times=int(lp["times"]), inject=True, inject_mode="step") if lp else None
    first = blocks[0].wattn
    ffs = [b.mlp.ff for b in blocks if b.mlp is not None]
    return ReaLModelConfig(
        n_layers=len(blocks), n_kv_heads=first.n_kv_heads, n_q_heads=first.n_heads, hidden_dim=int(d["width"]),
        intermediate_dim=max(ffs) if ffs else 0, vocab_size=int(d["vocab"]), head_dim=first.qk_dim, n_positions=None, embd_pdrop=0.0,
        resid_pdrop=0.0, attn_pdrop=0.0, layer_norm_epsilon=float(d["norm"]["eps"]), activation_function="silu",
        scale_attn_by_inverse_layer_idx=False, scale_attn_weights=True, use_attention_bias=False, use_attn_proj_bias=False,
        use_mlp_bias=False, layer_norm_type="gemma", mlp_type=None, apply_rotary=False, tied_embedding=not is_critic, is_critic=is_critic,
        blocks=blocks, norm_groups=1, sandwich_norm=False, conv_taps=0, fp32_residual=True, loop=loop, parallel_ff=True)


def config_to_dict(cfg: ReaLModelConfig) -> dict:
    layers = []
    for b in cfg.blocks:
        w, dl = b.wattn, b.delta
        left = dict(dim=w.qk_dim, heads=w.n_heads, kv_heads=w.n_kv_heads, scale=w.scale, vdim=w.v_dim)
        if w.window is not None:
            left["mask"] = dict(size=w.window)
        right = dict(conv=dl.conv_taps, dim=dl.qk_dim, heads=dl.n_heads, kv_heads=dl.n_kv_heads, vdim=dl.v_dim)
        m = dict(left=left, right=right)
        if b.branch_norm:
            left.update(bias_max=w.bias_max, bias_rows=w.bias_rows)
            right.update(decay_rank=dl.decay_rank, gate_rank=dl.gate_rank)
        else:
            m.update(left_scale=b.branch_scales[0], right_scale=b.branch_scales[1])
            r = w.rotary
            if r is not None:
                left["rot"] = dict(base=r.base, dims=r.dims)
                if r.factor is not None:
                    left["rot"]["scaling"] = dict(factor=r.factor, fast=r.fast, original=r.original, slow=r.slow)
        layers.append(dict(mixer=m, mlp=dict(ff=b.mlp.ff, kind="dense") if b.mlp is not None else None, type="parallel" if b.branch_norm else "parallel_2"))
    out = dict(architecture="Nufatar", layers=layers, norm=dict(eps=cfg.layer_norm_epsilon), vocab=cfg.vocab_size, width=cfg.hidden_dim)
    if cfg.loop is not None:
        out["loop"] = dict(start=cfg.loop.start, stop=cfg.loop.stop, times=cfg.loop.times)
    return out


def _in_parts(b: BlockConfig) -> List[Tuple[Tuple[str, ...], Tuple[int, ...], int]]:
    """The sections of `attn.in.weight` in order: (checkpoint names, their rows, padding rows at the end)."""
    w, d = b.wattn, b.delta
    nqk, nv, H = d.n_kv_heads * d.qk_dim, d.n_heads * d.v_dim, d.n_heads
    pad = lambda n: -n % 8
    out = [(("left.q",), (w.n_heads * w.qk_dim,), 0), (("left.k",), (w.n_kv_heads * w.qk_dim,), 0)]
    if not w.kv_shared:
        out.append((("left.v",), (w.value_width,), 0))
    out += [(("right.q",), (nqk,), 0), (("right.k",), (nqk,), 0), (("right.v",), (nv,), 0)]
    if d.decay_rank:
        return out + [(("right.b",), (H,), pad(H)), (("right.a1",), (d.decay_rank,), pad(d.decay_rank)), (("right.g1",), (d.gate_rank,), pad(d.gate_rank))]
    return out + [(("right.g",), (nv,), 0), (("right.b", "right.a"), (H, H), pad(2 * H))]


_PLAIN = {"attn.ln.weight": "norm1", "attn.rel.weight": "mix.left.rel", "attn.sink.weight": "mix.left.sink", "attn.o.weight": "mix.left.o",
          "attn.out_l.weight": "mix.left.out", "attn.A_log.weight": "mix.right.A_log", "attn.dt_bias.weight": "mix.right.dt_bias",
          "attn.o_norm.weight": "mix.right.norm", "attn.o2.weight": "mix.right.o", "attn.out_r.weight": "mix.right.out", "mlp.down.weight": "mlp.down"}


def _sd_from_ckpt(sd: Dict[str, torch.Tensor], cfg: ReaLModelConfig) -> Dict[str, torch.Tensor]:
    from realhf_b200.models.sharding import delta_low_ranks
    out: Dict[str, torch.Tensor] = {}
    L = cfg.n_layers
    if "embed" in sd:
        out["0.wte.weight"] = sd["embed"]
    if "final.norm" in sd:
        out[f"{L}.ln_f.weight"] = sd["final.norm"]
    if cfg.loop is not None and "loop.step" in sd:
        out[f"{cfg.loop.start + 1}.loop_step.weight"] = sd["loop.step"]
    for i, b in enumerate(cfg.blocks):
        cp, rp, d = f"l{i}.", f"{i + 1}.", b.delta
        if cp + "norm1" not in sd:
            continue
        for name, ck in _PLAIN.items():
            if cp + ck in sd:
                out[rp + name] = sd[cp + ck]
        rows = []
        for names, _, pad in _in_parts(b):
            rows += [sd[f"{cp}mix.{n}"] for n in names]
            if pad:
                rows.append(rows[-1].new_zeros(pad, rows[-1].shape[1]))
        out[rp + "attn.in.weight"] = torch.cat(rows, 0)
        out[rp + "attn.conv.weight"] = torch.cat([sd[f"{cp}mix.right.{n}.conv"] for n in ("q", "k", "v")], 0)
        if d.low_rank_width:
            ra, rg = delta_low_ranks(d)
            a2, g2 = sd[cp + "mix.right.a2"], sd[cp + "mix.right.g2"]
            low = a2.new_zeros(d.low_rank_width, ra + rg)
            low[:a2.shape[0], :a2.shape[1]] = a2
            low[a2.shape[0]:, ra:ra + g2.shape[1]] = g2
            out[rp + "attn.low.weight"] = low
        if b.mlp is not None:
            out[rp + "mlp.gate_up.weight"] = torch.cat([sd[cp + "mlp.gate"], sd[cp + "mlp.up"]], 0)
    return out


def _sd_to_ckpt(sd: Dict[str, torch.Tensor], cfg: ReaLModelConfig) -> Dict[str, torch.Tensor]:
    from realhf_b200.models.sharding import delta_low_ranks
    out: Dict[str, torch.Tensor] = {}
    for k, v in sd.items():
        li, name = k.split(".", 1)
        li = int(li)
        if li == 0:
            out["embed"] = v
            continue
        if name in ("ln_f.weight", "loop_step.weight"):
            out["final.norm" if name == "ln_f.weight" else "loop.step"] = v
            continue
        if li > cfg.n_layers:                                   # a critic's head, a pipeline stage's copy of the tied embedding
            out["head" if cfg.is_critic else "embed"] = v
            continue
        cp, b = f"l{li - 1}.", cfg.blocks[li - 1]
        d = b.delta
        if name in _PLAIN:
            out[cp + _PLAIN[name]] = v
        elif name == "attn.in.weight":
            off = 0
            for names, sizes, pad in _in_parts(b):
                for n, rows in zip(names, sizes):
                    out[f"{cp}mix.{n}"] = v[off:off + rows]
                    off += rows
                off += pad
        elif name == "attn.conv.weight":
            nqk = d.n_kv_heads * d.qk_dim
            for n, t in zip(("q", "k", "v"), torch.split(v, [nqk, nqk, d.n_heads * d.v_dim], 0)):
                out[f"{cp}mix.right.{n}.conv"] = t
        elif name == "attn.low.weight":
            ra = delta_low_ranks(d)[0]
            out[cp + "mix.right.a2"], out[cp + "mix.right.g2"] = v[:d.n_decays, :d.decay_rank], v[d.n_decays:, ra:ra + d.gate_rank]
        elif name == "mlp.gate_up.weight":
            out[cp + "mlp.gate"], out[cp + "mlp.up"] = v[:b.mlp.ff], v[b.mlp.ff:]
        else:
            raise KeyError(k)
    return {k: v.contiguous() for k, v in out.items()}


def _block_names(cfg: ReaLModelConfig, i: int) -> List[str]:
    b, cp = cfg.blocks[i], f"l{i}."
    names = [f"{cp}mix.{n}" for part in _in_parts(b) for n in part[0]] + [f"{cp}mix.right.{n}.conv" for n in ("q", "k", "v")]
    names += [cp + n for n in ("norm1", "mix.left.o", "mix.right.A_log", "mix.right.dt_bias", "mix.right.norm", "mix.right.o")]
    if b.branch_norm:
        names += [f"{cp}mix.{n}" for n in ("left.rel", "left.sink", "left.out", "right.a2", "right.g2", "right.out")]
    if b.mlp is not None:
        names += [cp + "mlp." + n for n in ("gate", "up", "down")]
    if cfg.loop is not None and i == cfg.loop.start:
        names.append("loop.step")
    if i == cfg.n_layers - 1:
        names.append("final.norm")
    return names


def make_test_config() -> ReaLModelConfig:
    par = dict(type="parallel", mlp=dict(kind="dense", ff=40),
               mixer=dict(left=dict(bias_max=20, bias_rows=8, dim=12, heads=4, kv_heads=2, vdim=12, scale=0.3, mask=dict(size=7)),
                          right=dict(conv=3, dim=8, heads=4, kv_heads=2, vdim=12, decay_rank=5, gate_rank=7)))
    par2 = dict(type="parallel_2", mlp=None,
                mixer=dict(left=dict(dim=8, heads=3, kv_heads=1, vdim=20, scale=0.4,
                                     rot=dict(base=300.0, dims=6, scaling=dict(factor=4.0, fast=8.0, original=64, slow=1.0))),
                           left_scale=0.7, right=dict(conv=4, dim=12, heads=2, kv_heads=1, vdim=8), right_scale=1.2))
    return config_from_dict(dict(layers=[par2, par, par2], loop=dict(start=1, stop=3, times=2), norm=dict(eps=1e-5), vocab=96, width=32))


register_hf_family(
    "nufatar", "Nufatar", lambda hf, is_critic=False: config_from_dict(hf if isinstance(hf, dict) else hf.to_dict(), is_critic),
    config_to_dict, _sd_from_ckpt, _sd_to_ckpt, lambda cfg: ["embed"], _block_names, lambda cfg: ["head"],
    make_test_config=make_test_config, config_from_dict=config_from_dict, config_to_dict=config_to_dict, weight_file="model.safetensors",
    config_from_shapes=config_from_shapes)
