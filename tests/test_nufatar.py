"""Nufatar (one norm per block, mixer and feed-forward side by side; attention over shared keys and values with a learned distance
bias, a window and a sink beside a delta rule with one decay per key channel, each side normalised; YaRN-rotated attention beside a
delta rule with one decay per head; a looped range with a learned vector per pass; tied embedding) against the plain float64
implementation in `nufatar_oracle.py`.

Every test body runs on the CPU (the op layer's PyTorch references, part of the default suite) and, marked `gpu`, on CUDA (the
sm_100a kernels) in fp32 and bf16.  Configurations are small and made here; none is a released model's."""

import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import nufatar_oracle as O
from realhf_b200.api.model import DeltaRuleConfig, GenerationHyperparameters, RotaryConfig, WindowAttentionConfig
from realhf_b200.models import generation as gen
from realhf_b200.models import hf_io
from realhf_b200.models.hetero_block import packed_meta
from realhf_b200.models.real_model import ReaLModel

F64 = torch.float64
CPU = pytest.param("cpu", torch.float32, id="cpu-f32")
GPU32 = pytest.param("cuda", torch.float32, id="cuda-f32", marks=pytest.mark.gpu)
GPU16 = pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=pytest.mark.gpu)
ALL = [CPU, GPU32, GPU16]
EXACT = [CPU, GPU32]


@pytest.fixture(autouse=True)
def one_thread():
    """Thousands of tiny CPU operations: a thread pool only slows them down."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def tol(dtype):
    return 2e-4 if dtype == torch.float32 else 0.05


def row_errs(got, want):
    """Per row: root mean square of the difference (mean removed) over the last dim, relative to the spread of `want`."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.double().std(-1).clamp_min(1e-6)).reshape(-1)


def worst(errs):
    return float(torch.cat([e.reshape(-1) for e in errs]).max()) if isinstance(errs, (list, tuple)) else float(errs.max())


def rounds_well(errs, dtype, share=0.02):
    """fp32: every row within the tolerance.  16 bit: all but a share of the rows; rows where a side's output nearly vanishes before its
    norm, or a query before its unit norm, lose digits to the operand type (the CPU references in bf16 lose the same)."""
    errs = torch.cat([e.reshape(-1) for e in errs])
    if dtype == torch.float32:
        return float(errs.max()) < tol(dtype)
    return float(errs.median()) < 0.03 and float((errs > tol(dtype)).float().mean()) <= share and float(errs.max()) < 0.5


def build(cfg: dict, w: dict, device, dtype) -> ReaLModel:
    fam = hf_io.family("nufatar")
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


def par(heads=4, kv_heads=2, dim=12, window=7, rows=8, bias_max=20, scale=None, r_heads=4, r_kv=2, r_dim=8, r_vdim=12, conv=3, ra=5, rg=7, mlp=None):
    left = dict(bias_max=bias_max, bias_rows=rows, dim=dim, heads=heads, kv_heads=kv_heads, scale=scale or dim ** -0.5, vdim=dim)
    if window is not None:
        left["mask"] = dict(size=window)
    right = dict(conv=conv, dim=r_dim, heads=r_heads, kv_heads=r_kv, vdim=r_vdim, decay_rank=ra, gate_rank=rg)
    return dict(type="parallel", mixer=dict(left=left, right=right), mlp=mlp)


def par2(heads=3, kv_heads=1, dim=8, vdim=20, dims=6, base=300.0, scaling=True, scale=None, r_heads=2, r_kv=1, r_dim=12, r_vdim=8, conv=4, ls=0.7,
         rs=1.2, mlp=None):
    left = dict(dim=dim, heads=heads, kv_heads=kv_heads, scale=scale or dim ** -0.5, vdim=vdim)
    if dims:
        left["rot"] = dict(base=base, dims=dims)
        if scaling:
            left["rot"]["scaling"] = dict(factor=4.0, fast=8.0, original=64, slow=1.0)
    right = dict(conv=conv, dim=r_dim, heads=r_heads, kv_heads=r_kv, vdim=r_vdim)
    return dict(type="parallel_2", mixer=dict(left=left, left_scale=ls, right=right, right_scale=rs), mlp=mlp)


def model_cfg(layers, loop=None, width=32, vocab=96, eps=1e-5):
    out = dict(architecture="Nufatar", layers=layers, norm=dict(eps=eps), vocab=vocab, width=width)
    if loop is not None:
        out["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return out


CONFIGS = {
    # both mixers, sizes that differ from layer to layer, a layer without a feed-forward, a loop in the middle
    "mixed": lambda: model_cfg([par2(mlp=dense(40)), par(mlp=None), par2(heads=4, kv_heads=2, dim=12, vdim=6, dims=4, scaling=False, mlp=dense(16)),
                                par(window=3, heads=2, kv_heads=1, r_kv=4, mlp=dense())], loop=(1, 3, 3)),
    # everything that can be 1 is 1: one head, a window of one token, one tap, ranks of 1, one pass over the whole stack
    "ones": lambda: model_cfg([par(heads=1, kv_heads=1, window=1, r_heads=1, r_kv=1, conv=1, ra=1, rg=1, mlp=dense(8)),
                               par2(heads=1, kv_heads=1, r_heads=1, r_kv=1, conv=1, ls=1.0, rs=1.0)], loop=(0, 2, 1), width=16, vocab=40),
    # sizes that are not multiples of four or eight, the last layer looped, no loop-free layer behind it
    "odd": lambda: model_cfg([par(heads=6, kv_heads=2, dim=7, window=13, rows=6, bias_max=9, r_heads=3, r_kv=3, r_dim=5, r_vdim=9, conv=5, ra=3, rg=11, mlp=dense(13)),
                              par2(heads=5, kv_heads=5, dim=10, vdim=7, dims=10, r_heads=3, r_kv=1, r_dim=9, r_vdim=5, conv=2, mlp=dense(30))],
                             loop=(1, 2, 4), width=20, vocab=50),
    # wide heads, windows longer than every prompt, no loop
    "wide": lambda: model_cfg([par2(heads=2, kv_heads=1, dim=136, vdim=200, dims=136, r_dim=136, r_vdim=144, mlp=dense(64)),
                               par(heads=12, kv_heads=1, dim=48, window=500, rows=16, bias_max=40, r_dim=72, r_vdim=40, ra=17, rg=16)], width=48, vocab=64),
}


def one_layer(layer, width=32, vocab=64, **kw):
    return model_cfg([layer], width=width, vocab=vocab, **kw)


MECHANISMS = {
    "parallel": lambda: one_layer(par()),
    "parallel-no-window": lambda: one_layer(par(window=None)),
    "parallel-all-heads-own-keys": lambda: one_layer(par(heads=3, kv_heads=3, dim=16, r_heads=3, r_kv=3)),
    "parallel-many-heads": lambda: one_layer(par(heads=18, kv_heads=2, dim=5, window=30, rows=2, bias_max=3, r_heads=6, r_kv=1)),
    "parallel-long-bias": lambda: one_layer(par(rows=20, bias_max=200, window=40)),
    "parallel-wide-state": lambda: one_layer(par(r_heads=2, r_kv=1, r_dim=70, r_vdim=34, conv=8, ra=24, rg=8)),
    "parallel_2": lambda: one_layer(par2()),
    "parallel_2-full-rotation": lambda: one_layer(par2(dim=16, dims=16, vdim=16)),
    "parallel_2-unscaled": lambda: one_layer(par2(heads=4, kv_heads=4, dim=7, vdim=9, dims=2, scaling=False)),
    "parallel_2-no-rotation": lambda: one_layer(par2(dims=0)),
    "parallel_2-scales": lambda: one_layer(par2(ls=-0.4, rs=2.5, r_heads=4, r_kv=4, r_dim=16, r_vdim=24)),
    "feed-forward": lambda: one_layer(par(mlp=dense(56))),
    "feed-forward-odd": lambda: one_layer(par2(mlp=dense(11)), width=24),
    "loop": lambda: one_layer(par2(mlp=dense(16)), loop=(0, 1, 3)),
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
    want = [O.forward(w, cfg, s) for s in full]
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
    assert worst(errs) < tol(dtype), worst(errs)


TC_SHAPES = {
    # windows that end inside, on and beyond the 128-row tiles of the tensor-core kernel; bias tables shorter and longer than the window
    "shared-64-window88": lambda: par(heads=3, kv_heads=1, dim=64, window=88, rows=16, bias_max=60),
    "shared-128-window128": lambda: par(heads=4, kv_heads=2, dim=128, window=128, rows=32, bias_max=300),
    "shared-64-window129": lambda: par(heads=8, kv_heads=1, dim=64, window=129, rows=8, bias_max=30),
    "shared-64-no-window-short-bias": lambda: par(heads=2, kv_heads=2, dim=64, window=None, rows=8, bias_max=16),
    "shared-128-rep6": lambda: par(heads=6, kv_heads=1, dim=128, window=200, rows=24, bias_max=150),
    "64-64": lambda: par2(heads=4, kv_heads=2, dim=64, vdim=64, dims=64),
    "64-128-rep6": lambda: par2(heads=12, kv_heads=2, dim=64, vdim=128, dims=24),
    "64-128-rep8": lambda: par2(heads=8, kv_heads=1, dim=64, vdim=128, dims=16),
    "128-64": lambda: par2(heads=3, kv_heads=1, dim=128, vdim=64, dims=128, scaling=False),
    "128-128-rep12": lambda: par2(heads=12, kv_heads=1, dim=128, vdim=128, dims=32),
}


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("name", list(TC_SHAPES))
def test_head_shapes_of_the_tensor_core_and_streaming_kernels(device, dtype, name):
    """Head sizes of 64 / 128: in 16 bit the prompts run the tcgen05 kernel and decoding the streaming kernel (whole caches and, with
    long ones, split keys); sequences of 1, 130 and 298 tokens cross tiles and windows.  No wait of the kernel ran out."""
    cfg = one_layer(TC_SHAPES[name](), width=64)
    w = O.random_checkpoint(cfg, 21)
    m = build(cfg, w, device, dtype)
    V = cfg["vocab"]
    seqs = [toks(n, V, 20 + n) for n in (1, 130, 298)]
    more = 6
    full = [s + toks(more, V, 90 + len(s)) for s in seqs]
    want = [O.forward(w, cfg, s) for s in full]
    sess = gen.StepSession(m, max_len=320, n_slots=3)
    lg = sess.logits(sess.prefill(list(enumerate(seqs))))
    off, errs = 0, []
    for s, wl in zip(seqs, want):
        errs.append(row_errs(lg[off:off + len(s)], wl[:len(s)]))
        off += len(s)
    for k in range(more):
        lg = sess.logits(sess.decode([(i, full[i][len(seqs[i]) + k]) for i in range(3)]))
        errs += [row_errs(lg[i:i + 1], want[i][len(seqs[i]) + k][None]) for i in range(3)]
    assert rounds_well(errs, dtype), worst(errs)
    if device == "cuda":
        from realhf_b200.ops import lib
        assert lib().attn_wait_error() == 0


def test_values_that_are_keys_have_one_cache():
    cfg = one_layer(par())
    st = gen.DecodeState(build(cfg, O.random_checkpoint(cfg, 1), "cpu", torch.float32), 2, 16)
    assert st.v[0] is st.k[0] and st.k[0].shape[2] == 7 and isinstance(st.m[0], tuple)


# ------------------------------------------------------------------------------------------------ edges, made to show


def silenced(w, *ends):
    """The checkpoint with the named output projections at zero (the other side then speaks alone)."""
    return {k: torch.zeros_like(t) if k.endswith(ends) else t for k, t in w.items()}


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("mode", ["prompt", "decode"])
@pytest.mark.parametrize("size", [1, 6, 16])
def test_window_edge_one_token_off_changes_the_output(device, dtype, mode, size):
    """Sharp scores (large scale), the recurrent side silenced: a window one token shorter or longer moves the oracle's logits by far more
    than the tolerance.  Decoding passes the ring's border several times."""
    cfg = one_layer(par(window=size, scale=3.0))
    w = silenced(O.random_checkpoint(cfg, 5), "right.o")
    seq = toks(40, cfg["vocab"], 77)
    want = O.forward(w, cfg, seq)
    for other in (size - 1, size + 1):
        if other:
            c2 = copy.deepcopy(cfg)
            c2["layers"][0]["mixer"]["left"]["mask"]["size"] = other
            assert float(row_errs(O.forward(w, c2, seq)[18:], want[18:]).max()) > 0.05
    m = build(cfg, w, device, dtype)
    got = packed_logits(m, [seq]) if mode == "prompt" else decoded_logits(m, seq, 3, max_len=48)
    assert float(row_errs(got, want).max()) < tol(dtype)


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("mode", ["prompt", "decode"])
@pytest.mark.parametrize("cut", [2, 17, 25])
def test_token_outside_the_window_is_invisible_and_the_first_inside_visible(device, dtype, mode, cut):
    """Window of 9, the last query at position 25, the recurrent side silenced: changing token 16 leaves the last logits as they were,
    changing token 17 moves them."""
    cfg = one_layer(par(window=9), vocab=32)
    w = silenced(O.random_checkpoint(cfg, 15), "right.o")
    seq = toks(26, 32, 3)
    m = build(cfg, w, device, dtype)

    def last(s):
        return (packed_logits(m, [s]) if mode == "prompt" else decoded_logits(m, s, cut))[-1:]
    base = last(seq)
    assert float(row_errs(base, O.forward(w, cfg, seq)[-1:]).max()) < tol(dtype)
    for at, seen in ((16, False), (17, True)):
        s2 = list(seq)
        s2[at] = (s2[at] + 5) % 32
        moved = float(row_errs(last(s2), base.double().cpu()).max())
        assert (moved > 1e-3) if seen else (moved < 1e-6), (at, moved)


def last_logits(m, seq, mode, cut):
    return (packed_logits(m, [seq]) if mode == "prompt" else decoded_logits(m, seq, cut))[-1:]


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("mode", ["prompt", "decode"])
def test_one_far_key_among_hundreds(device, dtype, mode):
    """Queries of token 30 point at keys of token 31 (in the dimensions that are not rotated), whose score stands out by far: placed among
    the first tokens of 300 it takes over the last token's attention, in the oracle and equally here."""
    cfg = one_layer(par2(dim=12, dims=6, scale=1.0), vocab=32)
    w = silenced(O.random_checkpoint(cfg, 9, F64), "right.o")
    h = O.one_plus_norm(w["embed"], w["l0.norm1"], 1e-5)
    u = torch.zeros(12, dtype=F64)
    u[8:] = 2.0
    point = lambda at, heads: torch.outer(u, h[at] / h[at].dot(h[at])).repeat(heads, 1)
    w.update({"l0.mix.left.q": point(30, 3), "l0.mix.left.k": point(31, 1)})
    w = {k: t.float() for k, t in w.items()}
    m = build(cfg, w, device, dtype)
    seq = toks(300, 30, 5)
    seq[-1] = 30
    base = O.forward(w, cfg, seq)[-1:]
    assert float(row_errs(last_logits(m, seq, mode, 270), base).max()) < tol(dtype)
    for at in (0, 1, 3, 120, 268):
        s2 = list(seq)
        s2[at] = 31
        want = O.forward(w, cfg, s2)[-1:]
        assert float(row_errs(want, base).max()) > 0.1
        assert float(row_errs(last_logits(m, s2, mode, 270), want).max()) < tol(dtype)


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("mode", ["prompt", "decode"])
def test_first_tokens_reach_the_last_logits_through_the_states(device, dtype, mode):
    """200 tokens, decays close to one, small writes, attention silenced: one of the first tokens moves the last logits through the states
    of both delta rules, in the oracle and equally here."""
    cfg = model_cfg([par(ra=3), par2()], vocab=32)
    w = silenced(O.random_checkpoint(cfg, 9), "left.o")
    w = {k: t - 9.0 if k.endswith("dt_bias") else t * 0.1 if k.endswith("right.b") else t for k, t in w.items()}
    seq = toks(200, 32, 5)
    m = build(cfg, w, device, dtype)
    base = O.forward(w, cfg, seq)[-1:]
    assert float(row_errs(last_logits(m, seq, mode, 170), base).max()) < tol(dtype)
    moved = []
    for at in (0, 2):
        s2 = list(seq)
        s2[at] = (s2[at] + 7) % 32
        want = O.forward(w, cfg, s2)[-1:]
        moved.append(float(row_errs(want, base).max()))
        assert float(row_errs(last_logits(m, s2, mode, 170), want).max()) < tol(dtype)
    assert max(moved) > 1e-3, moved                            # the oracle sees the first tokens


def _without(name):
    """(patched oracle functions, changed checkpoint) with one mechanism taken out."""
    att, core, norm1, mix, freq, rot = O.attend, O.delta_core, O.one_plus_norm, O.rms_divide, O.frequencies, O.rotate_half
    same = lambda w: w
    flat = lambda w: {k: (t.double().mean(0, keepdim=True).expand_as(t).contiguous() if k.endswith("left.rel") else t) for k, t in w.items()}

    def other_pairs(x, r):
        n = r["dims"]
        perm = torch.cat([torch.arange(0, n, 2), torch.arange(1, n, 2), torch.arange(n, x.shape[-1])])
        return rot(x[..., perm], r)[..., torch.argsort(perm)]
    return {
        "sink": ({"attend": lambda *a: att(*a[:6], None)}, same),
        "bias-shape": ({}, flat),
        "scaling": ({"frequencies": lambda r: freq({k: v for k, v in r.items() if k != "scaling"})}, same),
        "factor": ({"frequencies": lambda r: (freq(r)[0], 1.0)}, same),
        "pairs": ({"rotate_half": other_pairs}, same),
        "channel-decay": ({"delta_core": lambda q, k, v, b, g: core(q, k, v, b, g.mean(-1, keepdim=True).expand_as(g))}, same),
        "decay": ({"delta_core": lambda q, k, v, b, g: core(q, k, v, b, torch.ones_like(g))}, same),
        "write-strength": ({"delta_core": lambda q, k, v, b, g: core(q, k, v, torch.ones_like(b), g)}, same),
        "gate": ({"sigmoid": lambda x: torch.ones_like(x)}, same),
        "one-plus": ({"one_plus_norm": lambda x, w, e: norm1(x, w - 1.0, e)}, same),
        "side-norm": ({}, lambda w: {k: t * 3.0 if k.endswith("left.o") else t for k, t in w.items()}),
        "loop-step": ({}, lambda w: {k: t * 0 if k == "loop.step" else t for k, t in w.items()}),
        "step-order": ({}, lambda w: {k: t.flip(0) if k == "loop.step" else t for k, t in w.items()}),
        "history": ({"short_conv_silu": lambda x, cw: O.silu(x * cw[:, -1])}, same),
    }[name]


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("name,kind", [("sink", "par"), ("bias-shape", "par"), ("channel-decay", "par"), ("decay", "par"), ("decay", "par2"),
                                       ("write-strength", "par"), ("gate", "par"), ("gate", "par2"), ("one-plus", "par"), ("scaling", "par2"),
                                       ("factor", "par2"), ("pairs", "par2"), ("loop-step", "par2"), ("step-order", "par"), ("history", "par"),
                                       ("history", "par2")])
def test_every_mechanism_moves_the_logits_and_is_followed(device, dtype, name, kind, monkeypatch):
    """The oracle without the mechanism is far from the oracle with it; the framework follows the latter, in a prompt and decoded."""
    cfg = one_layer(par(window=20, mlp=dense()) if kind == "par" else par2(dims=8, scale=1.5, mlp=dense()), loop=(0, 1, 2))
    w = O.random_checkpoint(cfg, 4)
    seq = toks(36, cfg["vocab"], 8)
    want = O.forward(w, cfg, seq)
    patches, change = _without(name)
    with monkeypatch.context() as mp:
        for attr, fn in patches.items():
            mp.setattr(O, attr, fn)
        other = O.forward(change(w), cfg, seq)
    assert float(row_errs(other, want).max()) > 0.02
    m = build(cfg, w, device, dtype)
    assert float(row_errs(packed_logits(m, [seq]), want).max()) < tol(dtype)
    assert float(row_errs(decoded_logits(m, seq, 2), want).max()) < tol(dtype)


@pytest.mark.parametrize("device,dtype", EXACT)
def test_sides_are_normalised_before_they_are_halved(device, dtype):
    """Scaling one side's output projection changes nothing in `parallel` (its norm divides it out) and something in `parallel_2`."""
    for layer, moves in ((par(), False), (par2(), True)):
        cfg = one_layer(layer, eps=1e-9)
        w = O.random_checkpoint(cfg, 3)
        w2 = {k: t * 4.0 if k.endswith("left.o") else t for k, t in w.items()}
        seq = toks(20, cfg["vocab"], 1)
        a, b = (packed_logits(build(cfg, x, device, dtype), [seq]) for x in (w, w2))
        moved = float(row_errs(a, b.double().cpu()).max())
        assert (moved > 0.02) if moves else (moved < 1e-4)
        assert float(row_errs(b, O.forward(w2, cfg, seq)).max()) < tol(dtype)


def test_distance_buckets_match_the_formula():
    """Exact rows, logarithmic rows and the constant tail, for several table sizes and reaches (odd row counts among them)."""
    for B, D in ((8, 20), (32, 240), (2, 3), (16, 9), (7, 40), (40, 1000)):
        a = WindowAttentionConfig(n_heads=1, n_kv_heads=1, qk_dim=4, v_dim=4, scale=1.0, value_norm=False, slope_base=None, bias_rows=B, bias_max=D)
        t = a.distance_buckets()
        want = [O.distance_bucket(n, B, D) for n in range(len(t) + 500)]
        assert t == want[:len(t)] and all(b == B - 1 for b in want[len(t):]) and t[-1] == B - 1 and sorted(t) == t and len(t) <= D + 1


@pytest.mark.parametrize("device,dtype", ALL)
def test_every_distance_reads_its_own_bias(device, dtype):
    """Scores that are all equal (zero queries), bias rows far apart: the weights are the biases'.  300 tokens, a table of 150 distances
    with and without a window, in the layout of the tensor-core kernel and in a small one."""
    from realhf_b200.ops import attention as A
    for d, window in ((64, None), (64, 200), (128, 140), (12, None), (12, 33)):
        a = WindowAttentionConfig(n_heads=2, n_kv_heads=1, qk_dim=d, v_dim=d, scale=1.0, window=window, qkv_bias=False, value_norm=False, head_temp=False,
                                  slope_base=None, sink=True, out_gate=False, kv_shared=True, bias_rows=24, bias_max=150)
        g = torch.Generator().manual_seed(d)
        rel = (2.5 * torch.randn(24, 2, generator=g)).to(dtype)
        sink = torch.tensor([0.5, -1.0]).to(dtype)
        L = 300
        x = torch.randn(L, 3 * d, generator=g).to(dtype)
        x[:, :2 * d] = 0
        cu = torch.tensor([0, L], device=device, dtype=torch.int32)
        pos = torch.arange(L, device=device, dtype=torch.int32)
        xd = x.to(device)
        got = A.sink_window_attention(xd, A.window_values(xd, a), a, None, sink.to(device), pos, cu, L, rel=rel.to(device))
        k = x[:, 2 * d:].double().view(L, 1, d)
        bias = rel.double()[torch.tensor([O.distance_bucket(n, 24, 150) for n in range(L)])]
        want = O.attend(x[:, :2 * d].double().view(L, 2, d), k, k, 1.0, window, bias, sink.double()).reshape(L, -1)
        assert float((got.double().cpu() - want).abs().max()) < (2e-5 if dtype == torch.float32 else 0.03)
        rows = a.cache_rows(L)
        kc = torch.zeros(2, 1, rows, d, device=device, dtype=dtype)
        n = L - 1                                              # the last token decoded against the cache of the others
        tok = torch.ones(L, dtype=torch.int32, device=device)
        A.window_prepare_(xd[:n], a, None, None, 1e-5, pos=pos[:n], k_cache=kc, v_cache=kc, tok_slot=tok[:n], remain=(n - 1 - pos[:n]).int())
        lens = torch.tensor([0, n], dtype=torch.int32, device=device)
        one = A.sink_window_decode_attention(xd[n:], a, None, sink.to(device), kc, kc, lens, torch.tensor([1], dtype=torch.int32, device=device), 1e-5,
                                             rel=rel.to(device))
        assert float((one.double().cpu() - want[n:]).abs().max()) < (2e-5 if dtype == torch.float32 else 0.03)


@pytest.mark.parametrize("device,dtype", EXACT)
def test_rotation_with_a_factor_at_far_positions(device, dtype):
    """`window_prepare_` alone: half layout, YaRN frequencies and factor, positions up to 3000, packed and step form, against float64."""
    from realhf_b200.ops import attention as A
    g = torch.Generator().manual_seed(1)
    pos = torch.tensor([0, 1, 2, 63, 64, 500, 2999], dtype=torch.int32)
    lens = torch.tensor([5, 2999, 64], dtype=torch.int32)
    slots = torch.tensor([1, 2, 1, 0, 2, 2, 0], dtype=torch.int32)
    for H, G, d, dv, dims in ((3, 1, 12, 8, 8), (2, 2, 10, 6, 10), (4, 2, 64, 128, 32)):
        rot = dict(base=700.0, dims=dims, scaling=dict(factor=8.0, fast=16.0, original=128, slow=2.0))
        a = WindowAttentionConfig(n_heads=H, n_kv_heads=G, qk_dim=d, v_dim=dv, scale=1.0, qkv_bias=False, value_norm=False, head_temp=False, slope_base=None,
                                  sink=False, out_gate=False,
                                  rotary=RotaryConfig(dims=dims, base=700.0, interleaved=False, factor=8.0, original=128, fast=16.0, slow=2.0))
        x = torch.randn(7, (H + G) * d + G * dv, generator=g)
        f, ms = O.frequencies(rot)
        assert ms > 1.2
        for kw, n in ((dict(pos=pos.to(device)), pos), (dict(cache_lens=lens.to(device), slots=slots.to(device)), lens[slots.long()])):
            y = x.clone().to(device)
            A.window_prepare_(y, a, None, None, 1e-5, **kw)
            y = y.double().cpu()
            qk = x[:, :(H + G) * d].double().view(7, H + G, d)
            ang = n.double().unsqueeze(1) * f
            cs, sn, h = (torch.cos(ang) * ms).unsqueeze(1), (torch.sin(ang) * ms).unsqueeze(1), dims // 2
            u, v = qk[..., :h], qk[..., h:dims]
            want = torch.cat([u * cs - v * sn, v * cs + u * sn, qk[..., dims:]], -1).reshape(7, -1)
            near = n < 100
            assert float((y[:, :(H + G) * d] - want).abs().max()) < 3e-3 and float((y[near, :(H + G) * d] - want[near]).abs().max()) < 3e-5
            assert torch.equal(y[:, (H + G) * d:], x[:, (H + G) * d:].double())


# ------------------------------------------------------------------------------------------------ delta rule with a decay per channel


def delta_case(H, G, d, dv, taps, T, seed, dtype):
    """Projection rows [q | k | v | b | first factors], second factors etc. of a low-rank delta rule, and the oracle's inputs per row."""
    from realhf_b200.models.sharding import delta_low_ranks, delta_sections
    dl = DeltaRuleConfig(n_heads=H, n_kv_heads=G, qk_dim=d, v_dim=dv, conv_taps=taps, decay_rank=5, gate_rank=9, gate="sigmoid")
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g).to(dtype)
    proj = rn(T, sum(delta_sections(dl)))
    low = rn(T, dl.low_rank_width)
    assert sum(delta_low_ranks(dl)) == 24
    return dl, proj, low, rn(dl.conv_channels, taps) * taps ** -0.5, (torch.log(0.2 + torch.rand(H, generator=g))).to(dtype), rn(H * d)


def delta_inputs(dl, proj, low, conv_w, A_log, dt_bias):
    """The oracle's recurrence inputs of one sequence, from the same rows."""
    T, H, G, d, dv = proj.shape[0], dl.n_heads, dl.n_kv_heads, dl.qk_dim, dl.v_dim
    C = dl.conv_channels
    y = O.short_conv_silu(proj[:, :C].double(), conv_w.double())
    q = O.unit(y[:, :G * d].view(T, G, d)) * d ** -0.5
    k = O.unit(y[:, G * d:2 * G * d].view(T, G, d))
    z = (low[:, :H * d].double() + dt_bias.double()).view(T, H, d)
    decay = torch.exp(-torch.exp(A_log.double()).view(1, H, 1) * torch.nn.functional.softplus(z))
    return q, k, y[:, 2 * G * d:].view(T, H, dv), O.sigmoid(proj[:, C:C + H].double()), decay


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("H,G,d,dv,taps", [(2, 1, 8, 16, 4), (3, 3, 20, 5, 1), (2, 2, 64, 64, 2), (4, 2, 96, 40, 3), (1, 1, 200, 24, 8), (2, 1, 300, 12, 4)])
def test_channel_decay_prompt_then_decoding(device, dtype, H, G, d, dv, taps):
    """Prepare and recurrence alone: packed prompts (long enough for the token-tiled kernel) into shuffled slots with stale content, then
    token-by-token steps from the state they left, against the oracle's recurrence over whole sequences."""
    from realhf_b200.ops import recurrent as R
    prompt, total, slots = [1, 2, 60, 19], [9, 12, 66, 25], [3, 0, 4, 1]
    dl, proj, low, conv_w, A_log, dt_bias = delta_case(H, G, d, dv, taps, sum(total), H + d + taps, dtype)
    starts = [sum(total[:i]) for i in range(4)]
    ins = [delta_inputs(dl, proj[s:s + n], low[s:s + n], conv_w, A_log, dt_bias) for s, n in zip(starts, total)]
    want = [O.delta_core(*x) for x in ins]
    conv_state = torch.zeros(5, taps - 1, dl.conv_channels, device=device)
    s_state = torch.full((5, H, d, dv), 9.0, device=device)
    cut = lambda t: torch.cat([t[s:s + p] for s, p in zip(starts, prompt)]).to(device)
    cu = torch.tensor([0] + prompt, device=device).cumsum(0).int()
    meta = packed_meta(cu, sum(prompt), torch.tensor(slots, dtype=torch.int32), None, max(prompt))
    dev = [t.to(device) for t in (conv_w, A_log, dt_bias)]
    u = R.delta_prepare(cut(proj), *dev, dl, meta.pos, conv_state, meta.tok_slot, meta.remain, low=cut(low))
    wu = torch.cat([torch.cat([t[:p].reshape(p, -1) for t in x], -1) for x, p in zip(ins, prompt)])
    assert float((u.double().cpu() - wu).abs().max()) < (5e-6 if dtype == torch.float32 else 2e-2)
    o = R.delta_rule_scan(u, dl, cu, s_state, meta.seq_slot)
    scale = max(float(x.abs().max()) for x in want)
    lim = (5e-5 if dtype == torch.float32 else 0.05) * max(scale, 1e-3)
    assert float((o.double().cpu() - torch.cat([x[:p] for x, p in zip(want, prompt)])).abs().max()) < lim
    at = list(prompt)
    while True:
        live = [i for i in range(4) if at[i] < total[i]]
        if not live:
            break
        pick = torch.tensor([starts[i] + at[i] for i in live])
        sl = torch.tensor([slots[i] for i in live], dtype=torch.int32, device=device)
        u = R.delta_prepare_step(proj[pick].to(device), *dev, dl, conv_state, sl, low=low[pick].to(device))
        o = R.delta_rule_step(u, dl, s_state, sl)
        assert float((o.double().cpu() - torch.stack([want[i][at[i]] for i in live])).abs().max()) < lim
        for i in live:
            at[i] += 1
    assert bool((s_state[2] == 9.0).all())                    # a slot of nobody


@pytest.mark.parametrize("device,dtype", ALL)
def test_head_norm_with_either_gate(device, dtype):
    from realhf_b200.ops import recurrent as R
    g = torch.Generator().manual_seed(2)
    for T, H, dv, off in ((5, 3, 8, 0), (7, 2, 33, 3), (3, 1, 260, 8)):
        o = torch.randn(T, H, dv, generator=g)
        w = (1 + 0.3 * torch.randn(dv, generator=g)).to(dtype)
        row = torch.randn(T, H * dv + 8, generator=g).to(dtype)
        gate = row[:, off:off + H * dv]
        n = O.rms_divide(o.double(), 1e-5) * w.double()
        for act, f in (("silu", O.silu), ("sigmoid", O.sigmoid)):
            got = R.gated_head_norm(o.to(device), w.to(device), row.to(device)[:, off:off + H * dv], 1e-5, dtype, act)
            want = n.reshape(T, -1) * f(gate.double())
            assert float((got.double().cpu() - want).abs().max()) < (2e-5 if dtype == torch.float32 else 0.05)


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("T,W", [(1, 16), (5, 102), (37, 2050), (300, 4096), (3, 8192)])
def test_branch_sum_and_next_norm(device, dtype, T, W):
    """The sum of two normalised sides, a feed-forward and a vector into the fp32 stream with the next norm, every part optional; branch
    outputs as slices of wider rows at any alignment."""
    from realhf_b200.ops import functional as OF
    if device == "cpu" and T * W > 100000:
        pytest.skip("same code as the smaller sizes")
    g = torch.Generator().manual_seed(T + W)
    x = torch.randn(T, W, generator=g) * 3
    wide = torch.randn(T, 3 * W + 8, generator=g).to(dtype)
    vec = [(1 + 0.3 * torch.randn(W, generator=g)).to(dtype) for _ in range(4)]
    for use in ((1, 1, 1, 1, 1, 1), (1, 1, 1, 0, 0, 0), (1, 0, 0, 0, 0, 1), (0, 0, 0, 0, 0, 1), (1, 1, 0, 1, 0, 0), (0, 0, 1, 0, 0, 0)):
        for off in (0, 3):
            ys = [wide[:, off + i * W: off + (i + 1) * W] if use[i] else None for i in range(3)]
            w1, w2, step, nw = vec[0] if use[3] else None, vec[1] if use[4] else None, vec[2] if use[5] else None, vec[3]
            dv = lambda t: t.to(device) if t is not None else None
            wd = wide.to(device)
            yd = [wd[:, off + i * W: off + (i + 1) * W] if use[i] else None for i in range(3)]
            res = x.clone().to(device)
            out = OF.branch_add_norm_(res, *yd, 1e-5, 0.5, -0.8, dv(w1), dv(w2), dv(step), dv(nw), 1.0, dtype)
            n = lambda y, w: (O.rms_divide(y.double(), 1e-5) * w.double() if w is not None else y.double()) if y is not None else 0.0
            want = x.double() + 0.5 * n(ys[0], w1) - 0.8 * n(ys[1], w2) + n(ys[2], None) + (step.double() if step is not None else 0.0)
            assert torch.allclose(res.double().cpu(), want, atol=2e-5, rtol=1e-5)
            t_ = 2e-5 if dtype == torch.float32 else 3e-2
            assert torch.allclose(out.double().cpu(), O.rms_divide(want, 1e-5) * (1 + nw.double()), atol=t_, rtol=t_)
            res2 = x.clone().to(device)
            assert OF.branch_add_norm_(res2, *yd, 1e-5, 0.5, -0.8, dv(w1), dv(w2), dv(step)) is None and torch.equal(res2, res)


# ------------------------------------------------------------------------------------------------ whole models


@pytest.mark.parametrize("device,dtype", EXACT)
def test_long_decoding(device, dtype):
    """400 tokens, token by token from a 2-token prompt: a ring of 7 rows that is overwritten dozens of times, a cache that keeps
    everything and states that fade, in a loop, against the whole-sequence oracle."""
    cfg = model_cfg([par(window=7), par2(scaling=False)], loop=(0, 1, 2), vocab=32)
    w = O.random_checkpoint(cfg, 2)
    seq = toks(400, 32, 1)
    m = build(cfg, w, device, dtype)
    assert float(row_errs(decoded_logits(m, seq, 2), O.forward(w, cfg, seq)).max()) < tol(dtype)


@pytest.mark.parametrize("device,dtype", ALL)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_packed_forward_matches_oracle_layer_by_layer(device, dtype, name):
    cfg = CONFIGS[name]()
    w = O.random_checkpoint(cfg, 7)
    m = build(cfg, w, device, dtype)
    seqs = [toks(n, cfg["vocab"], 30 + n) for n in (23, 1, 6)]
    trace = []
    plain, got = packed_logits(m, seqs), packed_logits(m, seqs, trace=trace)
    assert float((plain.float() - got.float()).abs().max()) <= (1e-4 if dtype == torch.float32 else 0.1)
    off, errs = 0, []
    for s in seqs:
        want, wtr = O.forward(w, cfg, s, True)
        errs.append(row_errs(got[off:off + len(s)], want))
        assert len(trace) == len(wtr) == len(O.run_order(cfg))
        if dtype == torch.float32:
            for a, b in zip(trace, wtr):
                assert float((a[off:off + len(s)].double().cpu() - b).abs().max()) < 1e-4 * max(1.0, float(b.abs().max()))
        off += len(s)
    assert worst(errs) < tol(dtype), worst(errs)


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
    want = {r: O.forward(w, cfg, s) for r, s in full.items()}
    sess = gen.StepSession(m, max_len=96, n_slots=4)
    errs = []
    h = sess.prefill([(r, full[r][:plan[r][0]]) for r in plan])
    off = 0
    for r in plan:
        p = plan[r][0]
        errs.append(row_errs(sess.logits(h[off:off + p]), want[r][:p]))
        off += p
    late = {}
    for k in range(70):
        batch = [r for r in plan if k < plan[r][1]]
        lg = sess.logits(sess.decode([(r, full[r][plan[r][0] + k]) for r in batch]))
        errs += [row_errs(lg[j:j + 1], want[r][plan[r][0] + k][None]) for j, r in enumerate(batch)]
        done = [r for r in batch if k + 1 == plan[r][1]]
        if done:
            sess.release(done)
        if k == 25:                 # "b" and "d" have ended: two new requests reuse their slots while "a" and "c" go on
            late = {"e": (5, 30), "f": (1, 30)}
            for r, (p, n) in late.items():
                full[r] = toks(p + n, V, 70 + p)
                want[r] = O.forward(w, cfg, full[r])
            h = sess.prefill([(r, full[r][:late[r][0]]) for r in late])
            errs.append(row_errs(sess.logits(h[:5]), want["e"][:5]))
        for r in list(late):
            j = k - 26
            if 0 <= j < late[r][1]:
                lg = sess.logits(sess.decode([(r, full[r][late[r][0] + j])]))
                errs.append(row_errs(lg, want[r][late[r][0] + j][None]))
    assert rounds_well(errs, dtype, 0.15), worst(errs)


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
        assert float((together[off:off + len(s)] - alone).abs().max()) < 2e-4
        off += len(s)
    for cut in (1, 2, 7):
        assert float((decoded_logits(m, seqs[0], cut, max_len=40) - together[:30]).abs().max()) < 5e-4


@pytest.mark.parametrize("device,dtype", EXACT)
def test_session_grows_and_keeps_live_state(device, dtype):
    """More requests than slots: the state is re-allocated with twice the slots, the live requests' caches and states move."""
    cfg = CONFIGS["mixed"]()
    w = O.random_checkpoint(cfg, 14)
    m = build(cfg, w, device, dtype)
    V = cfg["vocab"]
    full = {r: toks(12 + r, V, 80 + r) for r in range(5)}
    want = {r: O.forward(w, cfg, s) for r, s in full.items()}
    sess = gen.StepSession(m, max_len=32, n_slots=2)
    sess.prefill([(r, full[r][:6]) for r in (0, 1)])
    sess.decode([(0, full[0][6]), (1, full[1][6])])
    sess.prefill([(r, full[r][:7]) for r in (2, 3, 4)])
    errs = []
    for k in range(7, 12):
        lg = sess.logits(sess.decode([(r, full[r][k]) for r in range(5)]))
        errs += [row_errs(lg[r:r + 1], want[r][k][None]) for r in range(5)]
    assert worst(errs) < tol(dtype), worst(errs)


@pytest.mark.parametrize("device,dtype", EXACT)
def test_greedy_generation_through_generate_and_inflight_batcher(device, dtype):
    cfg = CONFIGS["mixed"]()
    w = O.random_checkpoint(cfg, 6)
    m = build(cfg, w, device, dtype)
    n_new = 10
    prompts = [toks(n, cfg["vocab"], 50 + n) for n in (5, 1, 14)]
    want = [O.greedy(w, cfg, p, n_new) for p in prompts]
    g = GenerationHyperparameters(max_new_tokens=n_new, min_new_tokens=n_new, greedy=True, use_cuda_graph=(device == "cuda"))
    ids = torch.tensor([x for p in prompts for x in p], device=device)
    cu = torch.tensor([0] + [len(p) for p in prompts], device=device).cumsum(0).int()
    out, _ = gen.generate(m, ids, cu, g, eos_id=None, pad_id=0)
    assert out.tokens.tolist() == want
    ib = gen.InflightBatchingGenerator(m, g, eos_id=None, pad_id=0, n_slots=2, max_prompt_len=16)
    res = ib.generate([torch.tensor(p, device=device) for p in prompts])
    assert [r[0] for r in res] == want


def write_checkpoint(d, cfg, w):
    """As a checkpoint comes: the config without the sizes that only the tensors carry."""
    from safetensors.torch import save_file
    os.makedirs(d, exist_ok=True)
    bare = copy.deepcopy(cfg)
    for lay in bare["layers"]:
        for side, keys in (("left", ("bias_rows",)), ("right", ("decay_rank", "gate_rank"))):
            for k in keys:
                lay["mixer"][side].pop(k, None)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(bare, f)
    save_file({k: v.contiguous().bfloat16() for k, v in w.items()}, os.path.join(d, "model.safetensors"))
    return bare


def test_checkpoint_roundtrip_and_family_detection(tmp_path):
    """Sizes from the tensors' shapes, names both ways, the framework's own save and load, the parameter count."""
    fam = hf_io.family("nufatar")
    for name in ("mixed", "odd", "wide"):
        cfg = CONFIGS[name]()
        w = O.random_checkpoint(cfg, 8)
        d = str(tmp_path / name)
        bare = write_checkpoint(d, cfg, w)
        assert hf_io.family_of_path(d) == "nufatar"
        m = hf_io.from_hf("nufatar", d, dtype=torch.float32, device="cpu")
        assert fam.config_to_dict(m.config) == cfg and fam.config_from_shapes(bare, {k: tuple(t.shape) for k, t in w.items()}) == cfg
        assert sum(p.numel() for p in w.values()) == m.config.n_params()
        back = fam.sd_to_hf(m.state_dict(), m.config)
        assert set(back) == set(w) and all(torch.equal(back[k].float(), w[k].float()) for k in w)
        names = fam.embedding_param_names(m.config) + [n for i in range(m.config.n_layers) for n in fam.tblock_param_names(m.config, i)]
        assert set(names) == set(w)
        seq = toks(20, cfg["vocab"], 3)
        want = O.forward(w, cfg, seq)
        assert float(row_errs(packed_logits(m.eval(), [seq]), want).max()) < 2e-4
        d2 = str(tmp_path / (name + "-saved"))
        hf_io.save_to_hf(m, "nufatar", d2)
        m2 = hf_io.from_hf("nufatar", d2, dtype=torch.float32, device="cpu")
        assert float(row_errs(packed_logits(m2.eval(), [seq]), want).max()) < 2e-4


def test_configs_that_cannot_be_are_refused():
    fam = hf_io.family("nufatar")
    bad = [one_layer(dict(par(), type="parallel_3")), one_layer(par(mlp=dict(kind="moe", ff=8))), one_layer(par(rows=8, bias_max=4))]
    c = one_layer(par())
    c["layers"][0]["mixer"]["left"]["vdim"] = 16
    for cfg in bad + [c]:
        with pytest.raises(ValueError):
            fam.config_from_dict(cfg, False)


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
    wa, wb = O.forward(w, cfg, a), O.forward(w, cfg, b)
    want = {0: torch.stack([wa[0], wa[5], wb[1]]), 1: wb[2][None], 2: torch.stack([wa[7], wb[3]]), 3: wa[8][None]}
    for s, wl in want.items():
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{s}.f32"), dtype="<f4").reshape(-1, V))
        assert float(row_errs(got, wl).max()) < 2e-4


@pytest.mark.gpu
@pytest.mark.parametrize("rows", [1, 3, 200])
def test_projection_of_a_slice_at_any_offset(rows):
    """Column slices that start off a 16-byte boundary, one row among them (such a slice counts as contiguous)."""
    from realhf_b200.ops import functional as OF
    g = torch.Generator().manual_seed(rows)
    wide = torch.randn(rows, 88, generator=g).bfloat16().cuda()
    w = torch.randn(48, 32, generator=g).bfloat16().cuda()
    for off in (0, 3, 8, 20):
        for f in (OF.linear, OF.linear_f32):
            got = f(wide[:, off:off + 32], w)
            want = wide[:, off:off + 32].double() @ w.double().T
            assert float((got.double() - want).abs().max()) < 0.2
