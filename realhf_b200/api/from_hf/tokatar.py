"""Tokatar checkpoints <-> ReaLModel.

A Tokatar checkpoint is `config.json` + `model.safetensors`.  The config lists the layers one by one (`layers[i]` = mixer type
`attention`, `attention_2` or `latent_attention`, the mixer's sizes and constants, a dense feed-forward or null).  The model is a
heterogeneous stack (`ReaLModelConfig.blocks`) of mechanisms the config classes offer to any family:

  * a wrapped RMSNorm stack: norms before AND after every sublayer (`sandwich_norm`) with one learned factor each (`scalar_norm`), a
    learned vector on every branch output (`layer_scale`), the branch multiplied by sigmoid(W h + b) before its output norm
    (`gated_residual`), an fp32 residual stream, a constant on the embedding output (`embed_scale`);
  * `WindowAttentionConfig`, chunked, with an element-wise output gate (`element_gate`).  Mixer `attention`: half-layout rotation with
    "llama3" rescaled frequencies, soft-capped scores.  Mixer `attention_2`: biases, one RMS norm over all query (all key) heads
    (`full_norm`), interleaved rotation of queries, keys and values (`value_rotary`), one added to the softmax denominator
    (`sink_const` 0);
  * `LatentAttentionConfig` in its rotated form: half-layout rotation, no query latent, one output gate per head (`head_gate`);
  * `BlockMLPConfig(kind="relu2")`.

There is no `transformers` class for it: the config is read as a plain dict.

Checkpoint names -> framework names (layer i of the checkpoint is block i + 1 here):
  embed / head / final.norm                  0.wte.weight / {L+1}.head.weight / {L}.ln_f.weight [1]
  l<i>.norm1, norm1b, ls1                    attn.ln.weight [1], attn.ln_post.weight [1], attn.ls.weight
  l<i>.norm2, norm2b, ls2                    mlp.ln.weight [1], mlp.ln_post.weight [1], mlp.ls.weight
  mlp.up, rg2 / rg2.b                        mlp.up_rg.weight (sections [up | gate]) / mlp.up_rg.bias (zeros before the gate's)
  mlp.down                                   mlp.down.weight
  attention(_2): mix.q, k, v, g, rg1         attn.qkvg.weight (sections [q | k | v | g | residual gate])
                 mix.q.b, k.b, v.b, rg1.b    attn.qkvg.bias (zeros where the checkpoint has no bias)
                 mix.q.norm, k.norm / o      attn.q_norm.weight, attn.k_norm.weight / attn.o.weight
  latent_attention: mix.dkv, g, q, rg1       attn.in.weight (sections [latent, rotated key part | g | q | residual gate])
                 rg1.b                       attn.in.bias
                 mix.dkv.norm / uk, uv / o   attn.dkv_ln.weight / attn.ukv.weight / attn.o.weight
"""

from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from realhf_b200.api.model import (BlockConfig, BlockMLPConfig, LatentAttentionConfig, ReaLModelConfig, RotaryConfig, WindowAttentionConfig,
                                   register_hf_family)


def _rotary(rot: dict, interleaved: bool) -> RotaryConfig:
    sc = rot.get("scaling")
    kw = dict(scaling="llama3", factor=float(sc["factor"]), original=sc["original"], fast=float(sc["high"]), slow=float(sc["low"])) if sc else {}
    return RotaryConfig(dims=int(rot["dims"]), base=float(rot["base"]), interleaved=interleaved, **kw)


def _mlp_from_dict(i: int, f) -> Optional[BlockMLPConfig]:
    if f is None:
        return None
    if f.get("kind", "dense") != "dense":
        raise ValueError(f"Tokatar layer {i}: unknown feed-forward kind `{f['kind']}`")
    return BlockMLPConfig(kind="relu2", ff=int(f["ff"]))


def _mixer_from_dict(i: int, kind: str, m: dict) -> dict:
    if kind == "latent_attention":
        return dict(mixer="latent_attention", attn=LatentAttentionConfig(
            n_heads=int(m["heads"]), qk_dim=int(m["dim"]), v_dim=int(m["vdim"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
            rot_dim=int(m["rot_dim"]), rotary=_rotary(m["rot"], False), out_gate=True, head_gate=True))
    if kind not in ("attention", "attention_2"):
        raise ValueError(f"Tokatar layer {i}: unknown mixer type `{kind}`")
    second = kind == "attention_2"
    mask, vdim = m.get("mask"), int(m["vdim"])
    return dict(mixer="window_attention", wattn=WindowAttentionConfig(
        n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), qk_dim=int(m["dim"]), v_dim=vdim, scale=float(m["scale"]), window=None,
        keep_first=0, qkv_bias=second, value_norm=False, head_temp=False, slope_base=None, sink=False, out_gate=True, qk_norm=second,
        rotary=_rotary(m["rot"], second), chunk=int(mask["size"]) if mask else None,
        softcap=None if second or m.get("softcap") is None else float(m["softcap"]), sink_const=0.0 if second else None, element_gate=True,
        full_norm=second, value_rotary=RotaryConfig(dims=vdim, base=float(m["rot"]["base"]), interleaved=True) if second else None))


def config_from_dict(d: dict, is_critic: bool = False) -> ReaLModelConfig:
    blocks = [BlockConfig(mlp=_mlp_from_dict(i, lay.get("mlp")), **_mixer_from_dict(i, lay["type"], lay["mixer"])) for i, lay in enumerate(d["layers"])]
    first = blocks[0].wattn or blocks[0].attn
    ffs = [b.mlp.ff for b in blocks if b.mlp is not None]
    emb = d.get("embedding") or {}
    return ReaLModelConfig(
        n_layers=len(blocks), n_kv_heads=getattr(first, "n_kv_heads", first.n_heads), n_q_heads=first.n_heads, hidden_dim=int(d["width"]),
        intermediate_dim=max(ffs) if ffs else 0, vocab_size=int(d["vocab"]), head_dim=first.qk_dim, n_positions=None, embd_pdrop=0.0,
        resid_pdrop=0.0, attn_pdrop=0.0, layer_norm_epsilon=float(d["norm"]["eps"]), activation_function="relu",
        scale_attn_by_inverse_layer_idx=False, scale_attn_weights=True, use_attention_bias=False, use_attn_proj_bias=False,
        use_mlp_bias=False, layer_norm_type="rms", mlp_type=None, apply_rotary=False, tied_embedding=False, is_critic=is_critic,
        blocks=blocks, norm_groups=1, sandwich_norm=True, conv_taps=0, fp32_residual=True,
        embed_scale=float(emb["scale"]) if "scale" in emb else None, layer_scale=True, scalar_norm=True, gated_residual=True)


def _rot_to_dict(r: RotaryConfig) -> dict:
    out = dict(base=r.base, dims=r.dims)
    if r.factor is not None:
        out["scaling"] = dict(factor=r.factor, high=r.fast, low=r.slow, original=r.original)
    return out


def config_to_dict(cfg: ReaLModelConfig) -> dict:
    layers = []
    for b in cfg.blocks:
        if b.mixer == "latent_attention":
            a, kind = b.attn, "latent_attention"
            m = dict(dim=a.qk_dim, heads=a.n_heads, kv_rank=a.kv_rank, rot=_rot_to_dict(a.rotary), rot_dim=a.rot_dim, scale=a.scale, vdim=a.v_dim)
        else:
            a = b.wattn
            kind = "attention_2" if a.full_norm else "attention"
            m = dict(dim=a.qk_dim, heads=a.n_heads, kv_heads=a.n_kv_heads, rot=_rot_to_dict(a.rotary), scale=a.scale, vdim=a.v_dim)
            if a.chunk is not None:
                m["mask"] = dict(size=a.chunk)
            if a.softcap is not None:
                m["softcap"] = a.softcap
        layers.append(dict(mixer=m, mlp=dict(ff=b.mlp.ff, kind="dense") if b.mlp is not None else None, type=kind))
    out = dict(architecture="Tokatar", layers=layers, norm=dict(eps=cfg.layer_norm_epsilon), vocab=cfg.vocab_size, width=cfg.hidden_dim)
    if cfg.embed_scale is not None:
        out["embedding"] = dict(scale=cfg.embed_scale)
    return out


def _input_parts(cfg: ReaLModelConfig, i: int) -> Tuple[str, List[Tuple[str, Optional[str], int, int]]]:
    """(name of the fused input projection of layer i's mixer, its sections in order as (checkpoint weight, checkpoint bias or None,
    rows, rows with padding))."""
    from realhf_b200.models.sharding import in_sections
    b, cp = cfg.blocks[i], f"l{i}."
    sec = in_sections(cfg, i + 1)
    if b.mixer == "latent_attention":
        a = b.attn
        names = [("mix.dkv", None, a.cache_width), ("mix.g", None, a.n_heads), ("mix.q", None, a.n_heads * (a.qk_dim + a.rot_dim))]
    else:
        w = b.wattn
        bias = (lambda n: n + ".b") if w.qkv_bias else (lambda n: None)
        names = [("mix.q", bias("mix.q"), w.n_heads * w.qk_dim), ("mix.k", bias("mix.k"), w.n_kv_heads * w.qk_dim),
                 ("mix.v", bias("mix.v"), w.n_kv_heads * w.v_dim), ("mix.g", None, w.gate_width)]
    names.append(("rg1", "rg1.b", cfg.hidden_dim))
    return ("attn.in" if b.mixer == "latent_attention" else "attn.qkvg",
            [(cp + n, cp + nb if nb else None, rows, padded) for (n, nb, rows), padded in zip(names, sec)])


def _mlp_parts(cfg: ReaLModelConfig, i: int):
    F, cp = cfg.blocks[i].mlp.ff, f"l{i}."
    return [(cp + "mlp.up", None, F, (F + 7) // 8 * 8), (cp + "rg2", cp + "rg2.b", cfg.hidden_dim, cfg.hidden_dim)]


def _fuse(sd: Dict[str, torch.Tensor], parts) -> Tuple[torch.Tensor, torch.Tensor]:
    """Weight and bias of a fused projection: the sections' rows one after another, zero rows as padding, zeros for missing biases."""
    ws, bs = [], []
    for wn, bn, rows, padded in parts:
        w = sd[wn]
        ws += [w, w.new_zeros(padded - rows, w.shape[1])]
        bs += [sd[bn] if bn else w.new_zeros(rows), w.new_zeros(padded - rows)]
    return torch.cat(ws, 0), torch.cat(bs, 0)


_PLAIN = {"attn.ls.weight": "ls1", "mlp.ls.weight": "ls2", "attn.o.weight": "mix.o", "attn.q_norm.weight": "mix.q.norm",
          "attn.k_norm.weight": "mix.k.norm", "attn.dkv_ln.weight": "mix.dkv.norm", "mlp.down.weight": "mlp.down"}
_SCALAR = {"attn.ln.weight": "norm1", "attn.ln_post.weight": "norm1b", "mlp.ln.weight": "norm2", "mlp.ln_post.weight": "norm2b"}


def _plain_names(b: BlockConfig) -> List[str]:
    out = ["attn.ls.weight", "attn.o.weight"]
    if b.mixer == "latent_attention":
        out.append("attn.dkv_ln.weight")
    elif b.wattn.full_norm:
        out += ["attn.q_norm.weight", "attn.k_norm.weight"]
    return out + (["mlp.ls.weight", "mlp.down.weight"] if b.mlp is not None else [])


def _scalar_names(b: BlockConfig) -> List[str]:
    return list(_SCALAR) if b.mlp is not None else ["attn.ln.weight", "attn.ln_post.weight"]


def _sd_from_ckpt(sd: Dict[str, torch.Tensor], cfg: ReaLModelConfig) -> Dict[str, torch.Tensor]:
    out: Dict[str, torch.Tensor] = {}
    L = cfg.n_layers
    if "embed" in sd:
        out["0.wte.weight"] = sd["embed"]
    if "head" in sd:
        out[f"{L + 1}.head.weight"] = sd["head"]
    if "final.norm" in sd:
        out[f"{L}.ln_f.weight"] = sd["final.norm"].reshape(1)
    for i, b in enumerate(cfg.blocks):
        cp, rp = f"l{i}.", f"{i + 1}."
        if cp + "norm1" not in sd:
            continue
        for n in _scalar_names(b):
            out[rp + n] = sd[cp + _SCALAR[n]].reshape(1)
        for n in _plain_names(b):
            out[rp + n] = sd[cp + _PLAIN[n]]
        name, parts = _input_parts(cfg, i)
        out[rp + name + ".weight"], out[rp + name + ".bias"] = _fuse(sd, parts)
        if b.mixer == "latent_attention":
            out[rp + "attn.ukv.weight"] = torch.cat([sd[cp + "mix.uk"], sd[cp + "mix.uv"]], 0)
        if b.mlp is not None:
            out[rp + "mlp.up_rg.weight"], out[rp + "mlp.up_rg.bias"] = _fuse(sd, _mlp_parts(cfg, i))
    return out


def _sd_to_ckpt(sd: Dict[str, torch.Tensor], cfg: ReaLModelConfig) -> Dict[str, torch.Tensor]:
    out: Dict[str, torch.Tensor] = {}
    L = cfg.n_layers
    for k, v in sd.items():
        li, name = k.split(".", 1)
        li = int(li)
        if li == 0:
            out["embed"] = v
        elif li == L + 1:
            out["head"] = v
        elif name == "ln_f.weight":
            out["final.norm"] = v.reshape(())
        else:
            cp, b = f"l{li - 1}.", cfg.blocks[li - 1]
            if name in _PLAIN:
                out[cp + _PLAIN[name]] = v
            elif name in _SCALAR:
                out[cp + _SCALAR[name]] = v.reshape(())
            elif name == "attn.ukv.weight":
                n = b.attn.n_heads * b.attn.qk_dim
                out[cp + "mix.uk"], out[cp + "mix.uv"] = v[:n], v[n:]
            elif name.rsplit(".", 1)[0] in ("attn.in", "attn.qkvg", "mlp.up_rg"):
                parts = _mlp_parts(cfg, li - 1) if name.startswith("mlp") else _input_parts(cfg, li - 1)[1]
                off = 0
                for wn, bn, rows, padded in parts:
                    key = wn if name.endswith("weight") else bn
                    if key:
                        out[key] = v[off:off + rows]
                    off += padded
            else:
                raise KeyError(k)
    return {k: v.contiguous() for k, v in out.items()}


def _block_names(cfg: ReaLModelConfig, i: int) -> List[str]:
    b, cp = cfg.blocks[i], f"l{i}."
    parts = _input_parts(cfg, i)[1] + (_mlp_parts(cfg, i) if b.mlp is not None else [])
    names = [cp + _SCALAR[n] for n in _scalar_names(b)] + [cp + _PLAIN[n] for n in _plain_names(b)]
    names += [n for wn, bn, _, _ in parts for n in (wn, bn) if n]
    if b.mixer == "latent_attention":
        names += [cp + "mix.uk", cp + "mix.uv"]
    if i == cfg.n_layers - 1:
        names.append("final.norm")
    return names


def make_test_config() -> ReaLModelConfig:
    rot = dict(base=10000.0, dims=8)
    att = dict(type="attention", mlp=dict(kind="dense", ff=48),
               mixer=dict(dim=8, heads=4, kv_heads=2, vdim=12, scale=0.35, softcap=20.0, mask=dict(size=5),
                          rot=dict(rot, scaling=dict(factor=4.0, high=4.0, low=1.0, original=64))))
    att2 = dict(type="attention_2", mlp=None, mixer=dict(dim=12, heads=3, kv_heads=1, vdim=8, scale=0.3, mask=dict(size=7), rot=rot))
    lat = dict(type="latent_attention", mlp=dict(kind="dense", ff=40),
               mixer=dict(dim=8, heads=2, kv_rank=16, rot_dim=4, scale=0.3, vdim=12, rot=dict(base=5000.0, dims=4)))
    return config_from_dict(dict(layers=[att, att2, lat], norm=dict(eps=1e-5), embedding=dict(scale=4.0), vocab=96, width=32))


register_hf_family(
    "tokatar", "Tokatar", lambda hf, is_critic=False: config_from_dict(hf if isinstance(hf, dict) else hf.to_dict(), is_critic),
    config_to_dict, _sd_from_ckpt, _sd_to_ckpt, lambda cfg: ["embed"], _block_names, lambda cfg: ["head"],
    make_test_config=make_test_config, config_from_dict=config_from_dict, config_to_dict=config_to_dict, weight_file="model.safetensors")
