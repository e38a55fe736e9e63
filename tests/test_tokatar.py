"""Tokatar (heterogeneous wrapped RMSNorm stack: one factor per norm, layer scale, sigmoid-gated residuals; chunked attention with
rescaled rotation and soft-capped scores; chunked attention with a norm over all heads, turned values and one in the softmax
denominator; latent attention with a half-layout rotated key part and one gate per head; squared-relu feed-forwards) against the
plain float64 implementation in `tokatar_oracle.py`.

Every test body runs on the CPU (the op layer's PyTorch references, part of the default suite) and, marked `gpu`, on CUDA (the
sm_100a kernels) in fp32 and bf16.  Configurations are small and made here; none is a released model's."""

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import tokatar_oracle as O
from realhf_b200.api.model import GenerationHyperparameters, RotaryConfig, WindowAttentionConfig
from realhf_b200.models import generation as gen
from realhf_b200.models import hf_io
from realhf_b200.models.real_model import ReaLModel

CPU = pytest.param("cpu", torch.float32, id="cpu-f32")
GPU32 = pytest.param("cuda", torch.float32, id="cuda-f32", marks=pytest.mark.gpu)
GPU16 = pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=pytest.mark.gpu)
ALL = [CPU, GPU32, GPU16]
EXACT = [CPU, GPU32]


def tol(dtype):
    return 2e-4 if dtype == torch.float32 else 0.04


def row_errs(got, want):
    """Per row: root mean square of the difference (mean removed) over the last dim, relative to the spread of `want`."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.double().std(-1).clamp_min(1e-6)).reshape(-1)


def model_ok(errs, dtype):
    errs = torch.cat([e.reshape(-1) for e in errs]) if isinstance(errs, (list, tuple)) else errs
    return float(errs.max()) < tol(dtype)


def build(cfg: dict, w: dict, device, dtype) -> ReaLModel:
    fam = hf_io.family("tokatar")
    rc = fam.config_from_dict(cfg, False)
    m = ReaLModel(rc, dtype=dtype, device=device).instantiate(init="empty")
    m.load_state_dict(fam.sd_from_hf(w, rc))
    for p in m.parameters():
        p.requires_grad_(False)
    return m.eval()


def toks(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def packed_logits(m, seqs, trace=None):
    dev = m.device
    ids = torch.tensor([x for s in seqs for x in s], device=dev)
    cu = torch.tensor([0] + [len(s) for s in seqs], device=dev).cumsum(0).int()
    with torch.no_grad():
        if trace is not None:
            return m._forward_hetero(ids, cu, None, None, max(len(s) for s in seqs), trace=trace).logits
        return m(input_ids=ids, cu_seqlens=cu).logits


def decoded_logits(m, seq, cut, max_len=None):
    """The first `cut` tokens as a prompt, the rest one by one through the state: logits of every position."""
    sess = gen.StepSession(m, max_len=max_len or len(seq) + 1, n_slots=2)
    rows = [sess.logits(sess.prefill([("a", seq[:cut])]))]
    rows += [sess.logits(sess.decode([("a", t)])) for t in seq[cut:]]
    return torch.cat(rows)


# ------------------------------------------------------------------------------------------------ configurations

def dense(ff=24):
    return dict(ff=ff, kind="dense")


def att(heads=4, kv_heads=2, dim=12, vdim=8, chunk=5, dims=8, base=500.0, scaling=True, softcap=6.0, scale=None, mlp=None):
    rot = dict(base=base, dims=dims)
    if scaling:
        rot["scaling"] = dict(factor=4.0, high=3.0, low=1.5, original=48)
    m = dict(dim=dim, heads=heads, kv_heads=kv_heads, rot=rot, scale=scale or dim ** -0.5, softcap=softcap, vdim=vdim)
    if chunk is not None:
        m["mask"] = dict(size=chunk)
    return dict(type="attention", mixer=m, mlp=mlp)


def att2(heads=4, kv_heads=2, dim=8, vdim=12, chunk=7, dims=4, base=300.0, scale=None, mlp=None):
    m = dict(dim=dim, heads=heads, kv_heads=kv_heads, rot=dict(base=base, dims=dims), scale=scale or dim ** -0.5, vdim=vdim)
    if chunk is not None:
        m["mask"] = dict(size=chunk)
    return dict(type="attention_2", mixer=m, mlp=mlp)


def lat(heads=3, dim=8, vdim=12, kv_rank=16, rot_dim=4, base=200.0, scale=None, mlp=None):
    return dict(type="latent_attention", mlp=mlp, mixer=dict(dim=dim, heads=heads, kv_rank=kv_rank, rot=dict(base=base, dims=rot_dim),
                                                             rot_dim=rot_dim, scale=scale or (dim + rot_dim) ** -0.5, vdim=vdim))


def model_cfg(layers, width=32, vocab=96, eps=1e-5, embed_scale=3.0):
    return dict(architecture="Tokatar", embedding=dict(scale=embed_scale), layers=layers, norm=dict(eps=eps), vocab=vocab, width=width)


CONFIGS = {
    # all mixers, another order, a layer without a feed-forward, sizes that differ from layer to layer
    "mixed": lambda: model_cfg([lat(mlp=dense(40)), att2(mlp=None), att(mlp=dense(16)), att2(chunk=3, heads=2, kv_heads=1, mlp=dense()),
                                att(chunk=11, softcap=30.0, scaling=False, mlp=None)]),
    # everything that can be 1 is 1: one head, chunks of one token
    "ones": lambda: model_cfg([att(heads=1, kv_heads=1, chunk=1, mlp=dense(8)), att2(heads=1, kv_heads=1, chunk=1), lat(heads=1, mlp=dense(8))],
                              width=16, vocab=40, embed_scale=1.0),
    # sizes that are not multiples of four or eight, three heads per key head, feed-forwards of odd widths
    "odd": lambda: model_cfg([att2(heads=3, kv_heads=3, dim=10, vdim=6, dims=10, chunk=13, mlp=dense(13)), lat(heads=5, dim=7, vdim=9, kv_rank=11, rot_dim=6, mlp=dense(7)),
                              att(heads=6, kv_heads=2, dim=14, vdim=5, dims=6, chunk=9, mlp=dense(30))], width=20, vocab=50),
    # wide heads, chunks longer than every prompt
    "wide": lambda: model_cfg([att(heads=2, kv_heads=1, dim=136, vdim=200, dims=136, chunk=500, mlp=dense(64)),
                               lat(heads=2, dim=48, vdim=72, kv_rank=136, rot_dim=24, mlp=None), att2(heads=10, kv_heads=1, dim=16, vdim=144, dims=16, chunk=400)],
                              width=48, vocab=64),
}


def one_layer(layer, width=32, vocab=64, **kw):
    return model_cfg([layer], width=width, vocab=vocab, **kw)


MECHANISMS = {
    "attention": lambda: one_layer(att()),
    "attention-full-rotation": lambda: one_layer(att(dim=16, dims=16, vdim=16, chunk=6)),
    "attention-unscaled-odd": lambda: one_layer(att(heads=3, kv_heads=1, dim=7, vdim=9, dims=2, scaling=False, chunk=33)),
    "attention-tight-cap": lambda: one_layer(att(softcap=0.5, scale=2.0)),
    "attention-no-chunk": lambda: one_layer(att(chunk=None, dim=20, vdim=24, dims=20)),
    "attention_2": lambda: one_layer(att2()),
    "attention_2-all-heads-own-keys": lambda: one_layer(att2(heads=3, kv_heads=3, dim=16, vdim=16, dims=16, chunk=4)),
    "attention_2-odd": lambda: one_layer(att2(heads=5, kv_heads=1, dim=9, vdim=10, dims=6, chunk=21)),
    "attention_2-no-chunk": lambda: one_layer(att2(chunk=None, vdim=2)),
    "latent": lambda: one_layer(lat()),
    "latent-odd": lambda: one_layer(lat(heads=1, dim=5, vdim=7, kv_rank=9, rot_dim=2)),
    "latent-many-heads": lambda: one_layer(lat(heads=18, dim=4, vdim=6, kv_rank=20, rot_dim=8)),
    "feed-forward": lambda: one_layer(att(mlp=dense(56))),
    "feed-forward-odd": lambda: one_layer(att2(mlp=dense(11)), width=24, embed_scale=0.5),
}


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("name", list(MECHANISMS))
def test_mechanism_alone_prompt_then_decoding(device, dtype, name):
    """A one-layer model: packed prompts of unequal lengths (1 and 2 tokens among them) against the oracle, then the prompts'
    continuation token by token through the state the prefill left, in shuffled slots."""
    cfg = MECHANISMS[name]()
    w = O.random_checkpoint(cfg, 11)
    m = build(cfg, w, device, dtype)
    V = cfg["vocab"]
    seqs = [toks(n, V, 20 + n) for n in (1, 2, 37, 9)]
    more = 14
    full = [s + toks(more, V, 90 + len(s)) for s in seqs]
    want = [O.forward(cfg, w, s) for s in full]
    got = packed_logits(m, seqs)
    off, errs = 0, []
    for s, wl in zip(seqs, want):
        errs.append(row_errs(got[off:off + len(s)], wl[:len(s)]))
        off += len(s)
    sess = gen.StepSession(m, max_len=64, n_slots=6)
    sess.state.free_slots = [4, 1, 5, 0, 2, 3]
    h = sess.prefill(list(enumerate(seqs)))
    errs.append(row_errs(sess.logits(h[-1:]), want[-1][len(seqs[-1]) - 1][None]))
    for k in range(more):
        lg = sess.logits(sess.decode([(i, full[i][len(seqs[i]) + k]) for i in range(len(seqs))]))
        errs += [row_errs(lg[i:i + 1], want[i][len(seqs[i]) + k][None]) for i in range(len(seqs))]
    assert model_ok(errs, dtype), float(torch.cat(errs).max())


TC_SHAPES = {
    # chunk borders inside, on and beyond the 128-row tiles of the tensor-core kernel
    "cap-64-chunk88": lambda: one_layer(att(heads=3, kv_heads=1, dim=64, vdim=64, dims=64, chunk=88, softcap=8.0), width=64),
    "cap-128-chunk128": lambda: one_layer(att(heads=4, kv_heads=2, dim=128, vdim=128, dims=96, chunk=128), width=64),
    "cap-64-nochunk-rep8": lambda: one_layer(att(heads=8, kv_heads=1, dim=64, vdim=64, dims=32, chunk=None, softcap=20.0), width=64),
    "turned-64-chunk150": lambda: one_layer(att2(heads=2, kv_heads=2, dim=64, vdim=64, dims=64, chunk=150), width=64),
    "turned-128-chunk256-rep6": lambda: one_layer(att2(heads=6, kv_heads=1, dim=128, vdim=128, dims=32, chunk=256), width=64),
    "turned-64-chunk40": lambda: one_layer(att2(heads=2, kv_heads=1, dim=64, vdim=64, dims=64, chunk=40), width=64),
    "latent-64": lambda: one_layer(lat(heads=3, dim=48, rot_dim=16, vdim=64, kv_rank=72), width=64),
    "latent-128": lambda: one_layer(lat(heads=2, dim=96, rot_dim=32, vdim=128, kv_rank=160), width=64),
}


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("name", list(TC_SHAPES))
def test_head_shapes_of_the_tensor_core_and_streaming_kernels(device, dtype, name):
    """Head sizes 64 / 128 with equal query and value size: in 16 bit the prompts run the tcgen05 kernel and decoding the streaming
    kernel (whole caches and, with long ones, split keys); sequences of 1, 130 and 300 tokens cross tiles and chunks."""
    cfg = TC_SHAPES[name]()
    w = O.random_checkpoint(cfg, 21)
    m = build(cfg, w, device, dtype)
    V = cfg["vocab"]
    seqs = [toks(n, V, 20 + n) for n in (1, 130, 298)]
    more = 6
    full = [s + toks(more, V, 90 + len(s)) for s in seqs]
    want = [O.forward(cfg, w, s) for s in full]
    sess = gen.StepSession(m, max_len=320, n_slots=3)
    lg = sess.logits(sess.prefill(list(enumerate(seqs))))
    off, errs = 0, []
    for s, wl in zip(seqs, want):
        errs.append(row_errs(lg[off:off + len(s)], wl[:len(s)]))
        off += len(s)
    for k in range(more):
        lg = sess.logits(sess.decode([(i, full[i][len(seqs[i]) + k]) for i in range(3)]))
        errs += [row_errs(lg[i:i + 1], want[i][len(seqs[i]) + k][None]) for i in range(3)]
    assert model_ok(errs, dtype), float(torch.cat(errs).max())


# ------------------------------------------------------------------------------------------------ edges, made to show


def changed(cfg, layer=0, **kw):
    c2 = copy.deepcopy(cfg)
    c2["layers"][layer]["mixer"].update(kw)
    return c2


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("mode", ["prompt", "decode"])
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_chunk_border_one_token_off_changes_the_output(device, dtype, mode, kind):
    """Chunks of 6, sharp scores (large scale): a chunk of 5 or 7 picks other keys and moves the oracle's logits by far more than the
    tolerance.  Prompt and decoding forms are held against the oracle; decoding passes the chunk border six times, so every row of
    the ring is overwritten and a chunk starts over rows full of older keys."""
    cfg = one_layer(att(chunk=6, scale=4.0, softcap=40.0) if kind == "attention" else att2(chunk=6, scale=4.0))
    w = O.random_checkpoint(cfg, 5)
    seq = toks(40, cfg["vocab"], 77)
    want = O.forward(cfg, w, seq)
    for other in (5, 7):
        assert float(row_errs(O.forward(changed(cfg, mask=dict(size=other)), w, seq)[8:], want[8:]).max()) > 0.05
    m = build(cfg, w, device, dtype)
    got = packed_logits(m, [seq]) if mode == "prompt" else decoded_logits(m, seq, 3, max_len=48)
    assert float(row_errs(got, want).max()) < tol(dtype)


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("mode", ["prompt", "decode"])
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("cut", [12, 17])
def test_token_before_the_chunk_is_invisible_and_its_first_token_visible(device, dtype, mode, kind, cut):
    """Chunks of 9, the last query at position 25 (chunk 18 .. 26): changing token 17 leaves the last logits as they were, changing
    token 18 (the chunk's first) moves them; the decoding form starts at two different cuts, one right before the border."""
    cfg = one_layer(att(chunk=9) if kind == "attention" else att2(chunk=9), vocab=32)
    w = O.random_checkpoint(cfg, 15)
    seq = toks(26, 32, 3)
    m = build(cfg, w, device, dtype)

    def last(s):
        return (packed_logits(m, [s]) if mode == "prompt" else decoded_logits(m, s, cut))[-1:]
    base = last(seq)
    assert float(row_errs(base, O.forward(cfg, w, seq)[-1:]).max()) < tol(dtype)
    for at, seen in ((17, False), (18, True)):
        s2 = list(seq)
        s2[at] = (s2[at] + 5) % 32
        moved = float(row_errs(last(s2), base.double().cpu()).max())
        assert (moved > 1e-3) if seen else (moved < 1e-6), (at, moved)


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("mode", ["prompt", "decode"])
def test_far_key_dominates_through_the_latent_cache(device, dtype, mode):
    """300 tokens with sharp scores: changing one of the first tokens moves the last logits through the latent attention (in the
    oracle by more than 1e-3, and equally here), in a prompt and through 40 decoded tokens."""
    cfg = one_layer(lat(scale=3.0), vocab=32)
    w = O.random_checkpoint(cfg, 9)
    seq = toks(300, 32, 5)
    m = build(cfg, w, device, dtype)

    def last(s):
        return (packed_logits(m, [s]) if mode == "prompt" else decoded_logits(m, s, 260))[-1:]
    base = O.forward(cfg, w, seq)[-1:]
    assert float(row_errs(last(seq), base).max()) < tol(dtype)
    moved = []
    for at in range(4):
        s2 = list(seq)
        s2[at] = (s2[at] + 7) % 32
        want = O.forward(cfg, w, s2)[-1:]
        moved.append(float(row_errs(want, base).max()))
        assert float(row_errs(last(s2), want).max()) < tol(dtype)
    assert max(moved) > 1e-3                                   # the oracle sees the first tokens


def _without(name):
    """The oracle with one mechanism taken out (by patching the oracle's functions)."""
    saved = {}

    def patch(attr, fn):
        saved[attr] = getattr(O, attr)
        setattr(O, attr, fn)
    rot, attend, branch, freq = O.rotate, O.attend, O.branch, O.frequencies
    if name == "plus-one":
        patch("attend", lambda *a, plus_one=False, **k: attend(*a, **k))
    elif name == "softcap":
        patch("attend", lambda *a, softcap=None, **k: attend(*a, **k))
    elif name == "scaling":
        patch("frequencies", lambda r, n, scaled=True: freq(r, n, False))
    elif name == "turn-back":
        patch("rotate", lambda x, pos, f, inter: x if int(pos.min()) < 0 or (len(pos) > 1 and int(pos[-1]) < 0) else rot(x, pos, f, inter))
    elif name == "layout":
        patch("rotate", lambda x, pos, f, inter: rot(x, pos, f, not inter))
    elif name == "residual-gate":
        patch("branch", lambda x, sub, w, n, eps: branch(x, sub, dict(w, **{"rg" + n: w["rg" + n] * 0, f"rg{n}.b": w[f"rg{n}.b"] * 0}), n, eps))
    elif name == "layer-scale":
        patch("branch", lambda x, sub, w, n, eps: branch(x, sub, dict(w, **{"ls" + n: w["ls" + n] * 0 + 1}), n, eps))
    else:
        raise KeyError(name)

    def restore():
        for k, v in saved.items():
            setattr(O, k, v)
    return restore


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("name,layer", [("plus-one", "att2"), ("softcap", "att"), ("scaling", "att"), ("turn-back", "att2"), ("layout", "att"),
                                        ("layout", "att2"), ("layout", "lat"), ("residual-gate", "att"), ("layer-scale", "lat")])
def test_every_mechanism_moves_the_logits_and_is_followed(device, dtype, name, layer):
    """The oracle without the mechanism is far from the oracle with it; the framework follows the latter, in a prompt and decoded."""
    cfg = one_layer({"att": lambda: att(chunk=20, softcap=1.0, scale=1.0, mlp=dense()), "att2": lambda: att2(chunk=20, mlp=dense()),
                     "lat": lambda: lat(rot_dim=8, scale=1.0)}[layer]())
    w = O.random_checkpoint(cfg, 4)
    seq = toks(36, cfg["vocab"], 8)
    want = O.forward(cfg, w, seq)
    restore = _without(name)
    try:
        other = O.forward(cfg, w, seq)
    finally:
        restore()
    assert float(row_errs(other, want).max()) > 0.02
    m = build(cfg, w, device, dtype)
    assert float(row_errs(packed_logits(m, [seq]), want).max()) < tol(dtype)
    assert float(row_errs(decoded_logits(m, seq, 2), want).max()) < tol(dtype)


@pytest.mark.parametrize("device,dtype", ALL)
def test_large_scores_saturate_the_cap_and_the_unit_sink_stays_finite(device, dtype):
    """Scores far beyond the cap (all weights nearly equal) and far below zero (the added one holds nearly all the weight)."""
    for cfg in (one_layer(att(scale=60.0, softcap=2.0, chunk=30, dim=64, vdim=64, dims=64), width=64),
                one_layer(att2(scale=9.0, chunk=30, dim=64, vdim=64, dims=64), width=64)):
        w = O.random_checkpoint(cfg, 3)
        seq = toks(50, cfg["vocab"], 2)
        want = O.forward(cfg, w, seq)
        m = build(cfg, w, device, dtype)
        got = packed_logits(m, [seq])
        assert torch.isfinite(got).all()
        for lg in (got, decoded_logits(m, seq, 40)):
            errs = row_errs(lg, want)
            if dtype == torch.float32:
                assert float(errs.max()) < tol(dtype)
            else:                # one-hot softmax: 16-bit keys swap the weights of nearly equal scores in single rows
                assert float((errs > tol(dtype)).float().mean()) <= 0.2 and float(errs.median()) < 0.01


@pytest.mark.parametrize("device,dtype", EXACT)
def test_rotations_norms_and_turning_back_at_far_positions(device, dtype):
    """`window_prepare_` and `turn_gate_` alone: both layouts, part of a head and all of it, with and without the norm over all heads,
    positions up to 3000, packed and step form, against float64."""
    from realhf_b200.ops import attention as A
    g = torch.Generator().manual_seed(1)
    pos = torch.tensor([0, 1, 2, 63, 64, 500, 2999], dtype=torch.int32)
    lens = torch.tensor([5, 2999, 64], dtype=torch.int32)
    slots = torch.tensor([1, 2, 1, 0, 2, 2, 0], dtype=torch.int32)
    for H, G, d, dv, dims, inter, full in ((3, 1, 12, 8, 8, False, False), (2, 2, 10, 6, 10, True, True), (4, 2, 16, 24, 8, True, True),
                                           (1, 1, 7, 5, 2, False, False)):
        vr = RotaryConfig(dims=dv, base=50.0, interleaved=inter) if dv % 2 == 0 else None
        a = WindowAttentionConfig(n_heads=H, n_kv_heads=G, qk_dim=d, v_dim=dv, scale=1.0, chunk=4, qkv_bias=False, value_norm=False, head_temp=False,
                                  slope_base=None, sink=False, out_gate=True, element_gate=True, qk_norm=full, full_norm=full, value_rotary=vr,
                                  rotary=RotaryConfig(dims=dims, base=300.0, interleaved=inter))
        nq, nk, nv = H * d, G * d, G * dv
        x = torch.randn(7, nq + nk + nv + H * dv + 3, generator=g)
        wq, wk = 1 + 0.2 * torch.randn(nq, generator=g), 1 + 0.2 * torch.randn(nk, generator=g)
        f = O.frequencies(dict(base=300.0), dims)
        fv = O.frequencies(dict(base=50.0), dv) if vr else None

        def want_of(n):
            q, k, v = x[:, :nq].double(), x[:, nq:nq + nk].double(), x[:, nq + nk:nq + nk + nv].double().view(7, G, dv)
            if full:
                q, k = O.unit_rms(q, 1e-5) * wq.double(), O.unit_rms(k, 1e-5) * wk.double()
            q, k = O.rotate(q.view(7, H, d), n, f, inter), O.rotate(k.view(7, G, d), n, f, inter)
            return torch.cat([q.reshape(7, -1), k.reshape(7, -1), (O.rotate(v, n, fv, inter) if vr else v).reshape(7, -1)], -1)
        for kw, n in ((dict(pos=pos.to(device)), pos), (dict(cache_lens=lens.to(device), slots=slots.to(device)), lens[slots.long()])):
            y = x.clone().to(device)
            A.window_prepare_(y, a, wq.to(device), wk.to(device), 1e-5, **kw)
            y = y.double().cpu()
            want = want_of(n)
            near = n < 100
            assert float((y[:, :nq + nk + nv] - want).abs().max()) < 3e-3 and float((y[near, :nq + nk + nv] - want[near]).abs().max()) < 2e-5
            assert torch.equal(y[:, nq + nk + nv:], x[:, nq + nk + nv:].double())
            o = torch.randn(7, H * dv, generator=g)
            gate = x[:, nq + nk + nv:nq + nk + nv + H * dv]
            got = A.turn_gate_(o.clone().to(device), a, gate.to(device), **kw).double().cpu()
            back = O.rotate(o.double().view(7, H, dv), -n, fv, inter).reshape(7, -1) if vr else o.double()
            assert float((got - back * torch.sigmoid(gate.double())).abs().max()) < 3e-3


def test_frequency_scaling_has_three_bands():
    """Kept, blended and divided frequencies all occur and agree with the oracle's to 1e-12."""
    rot = dict(base=10000.0, dims=32, scaling=dict(factor=8.0, high=4.0, low=1.0, original=512))
    got, m = RotaryConfig(dims=32, base=10000.0, interleaved=False, factor=8.0, original=512, fast=4.0, slow=1.0, scaling="llama3").frequencies()
    want, plain = O.frequencies(rot, 32), O.frequencies(rot, 32, scaled=False)
    assert m == 1.0 and all(abs(a - b) < 1e-12 * b for a, b in zip(got, want))
    ratio = [a / b for a, b in zip(want, plain)]
    assert any(r == 1.0 for r in ratio) and any(abs(r - 0.125) < 1e-12 for r in ratio) and any(0.13 < r < 0.99 for r in ratio)


@pytest.mark.parametrize("device,dtype", EXACT)
def test_long_decoding_over_many_chunks(device, dtype):
    """400 tokens, token by token from a 2-token prompt: rings of 7 and 9 rows that are overwritten dozens of times beside a latent
    cache that keeps everything, against the whole-sequence oracle."""
    cfg = model_cfg([att(chunk=7), att2(chunk=9), lat()], vocab=32)
    w = O.random_checkpoint(cfg, 2)
    seq = toks(400, 32, 1)
    m = build(cfg, w, device, dtype)
    assert float(row_errs(decoded_logits(m, seq, 2), O.forward(cfg, w, seq)).max()) < tol(dtype)


# ------------------------------------------------------------------------------------------------ whole models


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_packed_forward_matches_oracle_layer_by_layer(device, dtype, name):
    cfg = CONFIGS[name]()
    w = O.random_checkpoint(cfg, 7)
    m = build(cfg, w, device, dtype)
    seqs = [toks(n, cfg["vocab"], 30 + n) for n in (23, 1, 6)]
    trace = []
    got = packed_logits(m, seqs, trace=trace)
    off, errs = 0, []
    for s in seqs:
        wtr = []
        want = O.forward(cfg, w, s, layers_out=wtr)
        errs.append(row_errs(got[off:off + len(s)], want))
        assert len(trace) == len(wtr)
        if dtype == torch.float32:
            for a, b in zip(trace, wtr):
                assert float((a[off:off + len(s)].double().cpu() - b).abs().max()) < 1e-4 * max(1.0, float(b.abs().max()))
        off += len(s)
    assert model_ok(errs, dtype), float(torch.cat(errs).max())


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_session_prefill_decode_batches_and_slot_reuse(device, dtype, name):
    """Unequal requests prefilled together, decoded together for 60+ steps while short ones end; new requests then take the freed
    slots (stale caches and states in them) and are checked from their first token on."""
    cfg = CONFIGS[name]()
    w = O.random_checkpoint(cfg, 8)
    m = build(cfg, w, device, dtype)
    V = cfg["vocab"]
    plan = {"a": (1, 64), "b": (2, 20), "c": (17, 70), "d": (9, 5)}          # prompt length, decoded tokens
    full = {r: toks(p + n, V, 40 + p) for r, (p, n) in plan.items()}
    want = {r: O.forward(cfg, w, s) for r, s in full.items()}
    sess = gen.StepSession(m, max_len=96, n_slots=4)
    errs = []
    h = sess.prefill([(r, full[r][:plan[r][0]]) for r in plan])
    off = 0
    for r in plan:
        p = plan[r][0]
        errs.append(row_errs(sess.logits(h[off:off + p]), want[r][:p]))
        off += p
    live = dict(plan)
    late = {}
    for k in range(70):
        batch = [r for r in live if k < live[r][1]]
        if not batch:
            break
        lg = sess.logits(sess.decode([(r, full[r][live[r][0] + k]) for r in batch]))
        errs += [row_errs(lg[j:j + 1], want[r][live[r][0] + k][None]) for j, r in enumerate(batch)]
        done = [r for r in batch if k + 1 == live[r][1]]
        if done:
            sess.release(done)
        if k == 25:                 # "b" and "d" have ended: two new requests reuse their slots while "a" and "c" go on
            late = {"e": (5, 30), "f": (1, 30)}
            for r, (p, n) in late.items():
                full[r] = toks(p + n, V, 70 + p)
                want[r] = O.forward(cfg, w, full[r])
            h = sess.prefill([(r, full[r][:late[r][0]]) for r in late])
            errs.append(row_errs(sess.logits(h[:5]), want["e"][:5]))
        for r in list(late):
            j = k - 25
            if k > 25 and j - 1 < late[r][1]:
                lg = sess.logits(sess.decode([(r, full[r][late[r][0] + j - 1])]))
                errs.append(row_errs(lg, want[r][late[r][0] + j - 1][None]))
    assert model_ok(errs, dtype), float(torch.cat(errs).max())


@pytest.mark.parametrize("device,dtype", EXACT)
def test_batched_equals_alone_and_prefill_equals_decoding(device, dtype):
    cfg = CONFIGS["mixed"]()
    w = O.random_checkpoint(cfg, 12)
    m = build(cfg, w, device, dtype)
    V = cfg["vocab"]
    seqs = [toks(n, V, 60 + n) for n in (30, 3, 11)]
    together = packed_logits(m, seqs)
    off = 0
    for s in seqs:
        alone = packed_logits(m, [s])
        assert float((together[off:off + len(s)] - alone).abs().max()) < 1e-4
        off += len(s)
    for cut in (1, 2, 7):
        assert float((decoded_logits(m, seqs[0], cut, max_len=40) - together[:30]).abs().max()) < 2e-4


@pytest.mark.parametrize("device,dtype", EXACT)
def test_session_grows_and_keeps_live_state(device, dtype):
    """More requests than slots: the state is re-allocated with twice the slots, the live requests' caches move."""
    cfg = CONFIGS["mixed"]()
    w = O.random_checkpoint(cfg, 14)
    m = build(cfg, w, device, dtype)
    V = cfg["vocab"]
    full = {r: toks(12 + r, V, 80 + r) for r in range(5)}
    want = {r: O.forward(cfg, w, s) for r, s in full.items()}
    sess = gen.StepSession(m, max_len=32, n_slots=2)
    sess.prefill([(r, full[r][:6]) for r in (0, 1)])
    sess.decode([(0, full[0][6]), (1, full[1][6])])
    sess.prefill([(r, full[r][:7]) for r in (2, 3, 4)])
    errs = []
    for k in range(7, 12):
        lg = sess.logits(sess.decode([(r, full[r][k]) for r in range(5)]))
        errs += [row_errs(lg[r:r + 1], want[r][k][None]) for r in range(5)]
    assert model_ok(errs, dtype), float(torch.cat(errs).max())


@pytest.mark.parametrize("device,dtype", EXACT)
def test_greedy_generation_through_generate_and_inflight_batcher(device, dtype):
    cfg = CONFIGS["mixed"]()
    w = O.random_checkpoint(cfg, 6)
    m = build(cfg, w, device, dtype)
    V, n_new = cfg["vocab"], 10
    prompts = [toks(n, V, 50 + n) for n in (5, 1, 14)]
    want = [O.greedy(cfg, w, p, n_new) for p in prompts]
    g = GenerationHyperparameters(max_new_tokens=n_new, min_new_tokens=n_new, greedy=True, use_cuda_graph=(device == "cuda"))
    ids = torch.tensor([x for p in prompts for x in p], device=device)
    cu = torch.tensor([0] + [len(p) for p in prompts], device=device).cumsum(0).int()
    out, _ = gen.generate(m, ids, cu, g, eos_id=None, pad_id=0)
    assert out.tokens.tolist() == want
    ib = gen.InflightBatchingGenerator(m, g, eos_id=None, pad_id=0, n_slots=2, max_prompt_len=16)
    res = ib.generate([torch.tensor(p, device=device) for p in prompts])
    assert [r[0] for r in res] == want


def write_checkpoint(d, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous().bfloat16() for k, v in w.items()}, os.path.join(d, "model.safetensors"))


def test_checkpoint_roundtrip_and_family_detection(tmp_path):
    for name in ("mixed", "odd"):
        cfg = CONFIGS[name]()
        w = O.random_checkpoint(cfg, 8)
        d = str(tmp_path / name)
        write_checkpoint(d, cfg, w)
        assert hf_io.family_of_path(d) == "tokatar"
        m = hf_io.from_hf("tokatar", d, dtype=torch.float32, device="cpu")
        fam = hf_io.family("tokatar")
        assert fam.config_to_dict(m.config) == cfg
        assert sum(p.numel() for p in w.values()) == m.config.n_params()
        back = fam.sd_to_hf(m.state_dict(), m.config)
        assert set(back) == set(w) and all(torch.equal(back[k].float(), w[k]) for k in w)
        seq = toks(20, cfg["vocab"], 3)
        assert float(row_errs(packed_logits(m.eval(), [seq]), O.forward(cfg, w, seq)).max()) < 2e-4


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=pytest.mark.gpu)])
def test_trace_replay_command(tmp_path, device):
    """`bin/trace_run` on a checkpoint directory: two requests prefilled in one step, decoded together, one ends early."""
    import numpy as np
    cfg = CONFIGS["mixed"]()
    w = O.random_checkpoint(cfg, 13)
    d = str(tmp_path / "ckpt")
    write_checkpoint(d, cfg, w)
    V = cfg["vocab"]
    a, b = toks(9, V, 1), toks(4, V, 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:6], want=[0, 5]), dict(id="b", tokens=b[:2], want=[1])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[6:7], want=[]), dict(id="b", tokens=b[2:3], want=[0])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[7:8], want=[0]), dict(id="b", tokens=b[3:4], want=[0])], end=["b"]),
             dict(step=3, entries=[dict(id="a", tokens=a[8:9], want=[0])], end=["a"])]
    out = str(tmp_path / "out")
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([sys.executable, exe, "--model", d, "--dtype", "float32", "--out", out, "--max-tokens", "32", "--device", device],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=1500)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    want = {0: torch.stack([wa[0], wa[5], wb[1]]), 1: wb[2][None], 2: torch.stack([wa[7], wb[3]]), 3: wa[8][None]}
    for s, wl in want.items():
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{s}.f32"), dtype="<f4").reshape(-1, V))
        assert float(row_errs(got, wl).max()) < 2e-4


# ------------------------------------------------------------------------------------------------ kernels against plain torch


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,W", [(1, 16), (5, 100), (37, 2050), (300, 4096)])
def test_gated_rms_norm_kernel_against_plain_torch(dtype, T, W):
    """RMSNorm with one factor, alone and fused with the gated, scaled residual add; the gate's logits are a column slice."""
    from realhf_b200.ops import functional as OF
    dev = torch.device("cuda:0")
    g = torch.Generator().manual_seed(T + W)
    x = (torch.randn(T, W, generator=g) * 3 + 1).to(dev)
    y = torch.randn(T, W, generator=g).to(dtype).to(dev)
    row = torch.randn(T, W + 24, generator=g).to(dtype).to(dev)
    ls = (1 + 0.3 * torch.randn(W, generator=g)).to(dtype).to(dev)
    w1, w2 = (torch.tensor([v]).to(dtype).to(dev) for v in (1.25, 0.75))
    tol_ = 1e-5 if dtype == torch.float32 else 2e-2
    assert torch.allclose(OF.centred_norm(x, w1, 1e-5, dtype, rms=True).double(), O.unit_rms(x.double(), 1e-5) * 1.25, atol=tol_, rtol=tol_)
    for gate in (row[:, 8:8 + W], row[:, 3:3 + W], None):
        res = x.clone()
        out = OF.residual_add_centred_norm_(res, y, w1, 1e-5, ls, 0.6, next_w=w2, out_dtype=dtype, rms=True, gate=gate)
        br = y.double() * (torch.sigmoid(gate.double()) if gate is not None else 1.0)
        want = x.double() + 0.6 * O.unit_rms(br, 1e-5) * 1.25 * ls.double()
        assert torch.allclose(res.double(), want, atol=1e-5, rtol=1e-5)
        assert torch.allclose(out.double(), O.unit_rms(want, 1e-5) * 0.75, atol=tol_, rtol=tol_)


@pytest.mark.gpu
@pytest.mark.parametrize("M,F,W,K", [(5, 24, 16, 32), (200, 104, 64, 64), (300, 512, 256, 192)])
def test_squared_relu_on_the_first_columns_only(M, F, W, K):
    """The up-projection with the residual gate's rows behind it: activation on the first F outputs, bias on all, small and large M."""
    from realhf_b200.ops import functional as OF
    dev = torch.device("cuda:0")
    g = torch.Generator().manual_seed(M)
    for dtype in (torch.float32, torch.bfloat16):
        x, w, b = (torch.randn(*s, generator=g).to(dtype).to(dev) for s in ((M, K), (F + W, K), (F + W,)))
        got = OF.relu2_linear(x, w, b, act_cols=F).double()
        z = x.double() @ w.double().T + b.double()
        want = torch.cat([torch.relu(z[:, :F]) ** 2, z[:, F:]], -1)
        rel = (got - want).abs() / want.abs().clamp_min(1.0)
        assert float(rel.max()) < (1e-4 if dtype == torch.float32 else 3e-2)
