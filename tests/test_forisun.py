"""The Forisun design in the library against the plain implementation of `plain_forisun.py`: small configurations made
here (sizes and options that differ from each other in every respect), random weights, every comparison on logits or on
one mechanism's output.  CPU tests cover the plain implementation itself, the configuration reader and the model
description; GPU tests cover the kernels one mechanism at a time and the engine: prompts, portions, single tokens,
unequal batches, slots and pages used again, far keys, the first tokens, long decoding, generation.  Prompt steps of the
bfloat16 engine have two ways through the mixer (as heads, in the latents' space); both are held to every case."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_forisun as P
from helpers import BF16_TOL, FP32_TOL, ROOT, random_tokens, rel_err


def tol_for(dtype):
    """The float32 engine is held to the library's float32 bound.  In bfloat16 the models here are 32 to 128 wide with
    peaked attention, and every sublayer's output passes a tanh of slope above 1: twice the library's bound (a key seen
    or missed by mistake moves these logits by far more; the cases below show it)."""
    return FP32_TOL if dtype == "float32" else 2 * BF16_TOL


def mixer(heads, dim, rot_dim, vdim, kv_rank, scale, base=1000.0, scaling=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale)
    if rot_dim:
        m["rot"] = dict(dims=rot_dim, base=base)
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, scale):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))


def layer(mix, mlp=None):
    return dict(type="latent_attention", mixer=mix, mlp=mlp)


def config(vocab, width, scale, layers, eps=1e-5):
    return dict(architecture="Forisun", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)


_YARN = (4.0, 64, 8.0, 1.0)
# own rows and rows of an earlier layer under other heads, key and value sizes; two layers that borrow from different
# places; experts, dense and none; scaled rotation in some layers
CFG_A = config(160, 64, 5.0, [
    layer(mixer(4, 16, 8, 24, 40, 0.5, 1000.0, _YARN), dense(96)),
    layer(mixer(3, 24, 4, 8, 40, 0.4, 50.0), moe(48, 6, 2, 1.7)),
    layer(mixer(2, 8, 8, 40, 40, 0.7, 1000.0, _YARN, kv_from=0)),
    layer(mixer(6, 16, 4, 16, 40, 0.4, 50.0, kv_from=1), moe(32, 5, 3, 0.6))])
# values that happen to be 1 or equal: one head, all sizes the same, one expert of one, a score scale and an embedding
# scale of 1, a weight scale of 1
CFG_B = config(200, 96, 1.0, [
    layer(mixer(1, 8, 8, 8, 8, 1.0, 50.0), moe(40, 1, 1, 1.0)),
    layer(mixer(8, 8, 8, 8, 8, 1.0, 50.0, kv_from=0), dense(8)),
    layer(mixer(1, 1, 2, 1, 24, 1.0, 10000.0), moe(64, 4, 1, 1.0)),
    layer(mixer(2, 16, 2, 16, 24, 0.3, 10000.0), dense(64))], eps=1e-6)
# sizes that are multiples of nothing: the bfloat16 products run on zero-padded operands, loads are scalar
CFG_C = config(75, 36, 3.0, [
    layer(mixer(3, 5, 6, 7, 11, 0.6, 100.0, (8.0, 32, 4.0, 1.0)), moe(13, 4, 2, 2.5)),
    layer(mixer(2, 9, 6, 19, 11, 0.5, 100.0, (8.0, 32, 4.0, 1.0), kv_from=0), dense(22)),
    layer(mixer(5, 3, 0, 6, 13, 0.6), moe(11, 7, 3, 0.8))])
# sizes that the tensor-core kernels take (the first layer's experts as grouped products): heads of 128 and of 192
# numbers, rows above and below the size from which a tile has 32 keys
CFG_D = config(128, 128, 11.0, [
    layer(mixer(8, 64, 64, 64, 256, 0.15, 250000.0, (16.0, 4096, 32.0, 1.0)), moe(128, 8, 2, 1.5)),
    layer(mixer(2, 128, 64, 128, 264, 0.12, 10000.0), dense(256)),
    layer(mixer(16, 32, 64, 32, 256, 0.2, 250000.0, (16.0, 4096, 32.0, 1.0), kv_from=0), None)])
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}
TAGS = 4          # features that carry a token's class for the routers (see `decisive`)


def bf(t):
    return t.to(torch.bfloat16).to(P.DT)


def decisive(cfg, w):
    """Routers whose choice no rounding turns: the last TAGS features of the residual stream carry the token's class
    (id mod TAGS) from the embedding, no sublayer writes them (the rows of every last product that would are zero, and
    so are the norms' biases there), and a router reads next to nothing else: every class has its own order of the
    experts with gaps between their scores (the norm in front has no bias there), and the corrections lift half of the experts above the others."""
    out = dict(w)
    W = cfg["width"]
    emb = w["embed"].clone()
    emb[:, W - TAGS:] = 0.0
    for tok in range(cfg["vocab"]):
        emb[tok, W - TAGS + tok % TAGS] = 4.0
    out["embed"] = emb
    for name in w:
        if name.endswith(".o") or name.endswith(".down"):
            t = w[name].clone()
            t[W - TAGS:] = 0.0
            out[name] = t
        if name.endswith(("b.b", "norm2.b")) or name == "embed.norm.b":
            t = w[name].clone()
            t[W - TAGS:] = 0.0
            out[name] = t
    for i, lay in enumerate(cfg["layers"]):
        if lay.get("mlp") is None or lay["mlp"]["kind"] != "moe":
            continue
        E = lay["mlp"]["router"]["experts"]
        r = bf(w[f"l{i}.mlp.router"] * 0.03)
        g = torch.Generator().manual_seed(1000 + i)
        for c in range(TAGS):
            order = torch.randperm(E, generator=g)
            r[order, W - TAGS + c] = bf(torch.linspace(-1.6, 1.6, E, dtype=P.DT))
        out[f"l{i}.mlp.router"] = r
        out[f"l{i}.mlp.correction"] = bf((torch.randperm(E, generator=g) % 2).to(P.DT) * 1.4 - 0.5)
    return out


def weights_for(cfg, seed):
    return decisive(cfg, P.random_weights(cfg, seed))


def folder(tmp_path, cfg, seed):
    w = weights_for(cfg, seed)
    return P.save_folder(cfg, w, str(tmp_path / f"model{seed}")), w


def plain_logits(cfg, w, ids):
    """The plain implementation's logits, with the check that no router's choice was a close call."""
    P.MARGINS.clear()
    out, _ = P.forward(cfg, w, list(ids))
    assert not P.MARGINS or min(P.MARGINS) > 0.01, min(P.MARGINS)
    return out


# ------------------------------------------------------------------------------------------------
# without a device
# ------------------------------------------------------------------------------------------------
def test_the_plain_implementation_gives_the_same_logits_in_pieces():
    for name, cfg in CONFIGS.items():
        w = weights_for(cfg, 3)
        ids = random_tokens(90, cfg["vocab"], 7)
        whole = plain_logits(cfg, w, ids)
        pieces = P.forward_in_pieces(cfg, w, ids, [1, 1, 2, 3, 60, 1, 22])
        assert float((whole - pieces).abs().max()) < 1e-9, name


def test_the_plain_mechanisms_follow_their_definitions_on_cases_done_by_hand():
    one = lambda *x: torch.tensor(x, dtype=P.DT)  # noqa: E731
    # dynamic tanh: ln(2) / 2 has tanh (2 - 1) / (2 + 1); weight and bias act feature by feature
    x = P.squash(one(math.log(2.0), 0.0), one(0.5), one(3.0, 7.0), one(0.25, -1.0))
    assert torch.allclose(x, one(1.25, -1.0))
    # the exact GELU: Phi(1) = 0.841344746...
    assert abs(float(P.gelu(one(1.0))) - 0.8413447460685429) < 1e-12 and float(P.gelu(one(0.0))) == 0.0
    # frequencies without scaling: base^(-2 i / dims)
    f, a = P.frequencies(dict(dims=4, base=100.0))
    assert torch.allclose(f, one(1.0, 0.1)) and a == 1.0
    # with scaling: pair(t) = dims ln(original / (2 pi t)) / (2 ln base).  base e^2, dims 8, original 2 pi e^6 gives
    # pair(1) = 8 * 6 / 4 = 12 -> hi = min(12, 7) = 7; pair(e^4) = 8 * 2 / 4 = 4 (lo); pairs 0..3 are kept whole
    sc = dict(factor=math.e ** 5, original=2 * math.pi * math.e ** 6, fast=math.e ** 4 * 1.0000001, slow=1.0)
    f, a = P.frequencies(dict(dims=8, base=math.e ** 2, scaling=sc))
    assert abs(a - 1.5) < 1e-12 and abs(float(f[2]) - math.e ** -1.0) < 1e-12     # lo = 3: ramp 0 up to pair 3
    assert abs(float(f[3]) - math.e ** -1.5) < 1e-12
    # fast = slow at pair 1.5: lo 1, hi 2; pair 0 and 1 keep their frequency, pairs 2 and 3 are divided by the factor
    sc = dict(factor=2.0, original=2 * math.pi * math.e ** 0.75, fast=1.0, slow=1.0)
    f, a = P.frequencies(dict(dims=8, base=math.e ** 2, scaling=sc))
    assert torch.allclose(f, one(1.0, math.e ** -0.5, 0.5 * math.e ** -1.0, 0.5 * math.e ** -1.5))
    # rotation pairs number i with i + dims / 2; base 1: every frequency is 1, the angle at position 1 is 1
    y = P.rotate(one(1.0, 2.0, 3.0, 4.0).view(1, 1, 4), torch.tensor([1]), dict(dims=4, base=1.0))
    c, s = math.cos(1.0), math.sin(1.0)
    assert torch.allclose(y.flatten(), one(1 * c - 3 * s, 2 * c - 4 * s, 3 * c + 1 * s, 4 * c + 2 * s))
    # attention sees the own position and the earlier ones: scores ln 3 and 0 weigh 3/4 and 1/4
    q, k = one(1.0, 1.0).view(2, 1, 1), one(math.log(3.0), 0.0).view(2, 1, 1)
    v = one(8.0, 4.0).view(2, 1, 1)
    assert torch.allclose(P.causal_attention(q, k, v, 0, 1.0).flatten(), one(8.0, 7.0))
    # the choice goes by sigmoid + correction, the weight is sigmoid * scale without it
    chosen, weight = P.choose_experts(one([0.0, 1.0, 2.0]).view(1, 3), one(0.9, 0.0, -0.9), 2, 2.0)
    assert chosen[0].tolist() == [0, 1]
    assert torch.allclose(weight[0], 2.0 * torch.sigmoid(one(0.0, 1.0)))
    # the weight multiplies the expert's output
    w = {"m.router": one([0.0], [1.0]), "m.correction": one(0.0, 0.0)}
    for x, k in (("e0", 1.0), ("e1", 3.0)):
        w[f"m.{x}.gate"], w[f"m.{x}.up"], w[f"m.{x}.down"] = one([1.0]), one([2.0]), one([k])
        w[f"m.{x}.gate"], w[f"m.{x}.up"], w[f"m.{x}.down"] = (t.view(1, 1) for t in (w[f"m.{x}.gate"], w[f"m.{x}.up"], w[f"m.{x}.down"]))
    h = one([1.5]).view(1, 1)
    base = P.silu(h) * 2.0 * h
    got = P.expert_ff(dict(router=dict(experts=2, top=2, scale=0.5)), w, "m.", h)
    assert torch.allclose(got, 0.5 * (0.5 * base + torch.sigmoid(one(1.5)) * 3.0 * base))


def test_configuration_is_read_by_key_and_written_back():
    from janus_b200.config import ConfigError, resolve_architecture
    for cfg in CONFIGS.values():
        arch = resolve_architecture(cfg)
        c = arch.config_class.from_dict(cfg)
        assert json.loads(json.dumps(c.to_dict())) == json.loads(json.dumps(cfg))
    arch = resolve_architecture(CFG_A)
    c = arch.config_class.from_dict(CFG_A)
    assert c.layers[2].mlp is None and c.layers[2].mixer.kv_from == 0 and c.layers[3].mixer.kv_from == 1
    assert c.layers[0].mixer.rot.scaling == (4.0, 64.0, 8.0, 1.0) and c.layers[1].mixer.rot.scaling is None
    assert c.layers[1].mlp.scale == 1.7 and c.embedding_scale == 5.0
    for path, value, word in ((("layers", 0, "type"), "attention", "type"), (("layers", 0, "mlp", "kind"), "sparse", "kind"),
                              (("norm",), None, "norm"), (("embedding",), None, "embedding"), (("layers",), [], "layers"),
                              (("layers", 0, "mixer", "rot", "dims"), 4, "dims"), (("layers", 0, "mixer", "rot"), None, "rot"),
                              (("layers", 0, "mixer", "kv_rank"), None, "kv_rank"),
                              (("layers", 1, "mlp", "router", "top"), 7, "top"),
                              (("layers", 2, "mixer", "kv_from"), 2, "kv_from"), (("layers", 3, "mixer", "kv_from"), 2, "kv_from"),
                              (("layers", 2, "mixer", "kv_rank"), 24, "kv_from"),
                              (("layers", 2, "mixer", "rot", "base"), 999.0, "kv_from"),
                              (("layers", 0, "mixer", "scale"), 0.0, "scale")):
        bad = copy.deepcopy(CFG_A)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            arch.config_class.from_dict(bad)


def test_the_model_description_names_every_tensor_once_and_places_read_the_rows_they_should():
    from janus_b200.config import resolve_architecture
    from janus_b200.models.forisun import forisun_spec
    for cfg in CONFIGS.values():
        arch = resolve_architecture(cfg)
        c = arch.config_class.from_dict(cfg)
        names = {s.name: tuple(s.shape) for s in arch.weight_specs(c)}
        want = {k: tuple(v.shape) for k, v in P.random_weights(cfg, 0).items()}
        assert names == want
    spec = forisun_spec(resolve_architecture(CFG_A).config_class.from_dict(CFG_A))
    assert [e.reads_cache_of for e in spec.schedule] == [None, None, 0, 1]
    assert spec.layers[2].feed_forward is None and "l2.norm2.alpha" in spec.ignorable_weights
    from janus_b200.engine.model import DecoderModel
    model = DecoderModel(spec, torch.bfloat16, torch.device("cpu"))
    specs = model.place_cache_specs()
    assert [s.head_dim if s else None for s in specs] == [48, 48, None, None]     # 40 + 8; 40 + 4, stored in 16-byte pieces
    assert DecoderModel(spec, torch.float32, torch.device("cpu")).place_cache_specs()[1].head_dim == 44


def test_rows_that_no_kernel_takes_are_refused_when_the_model_is_built():
    from janus_b200.parts.latent_attention import RotaryLatentAttention
    for dtype in (torch.float32, torch.bfloat16):
        RotaryLatentAttention(64, 2, 8, 64, 8, 1024, 1.0, 1e-5, dtype=dtype, device=torch.device("cpu"))
        with pytest.raises(ValueError, match="rows"):
            RotaryLatentAttention(64, 2, 8, 64, 8, 1280, 1.0, 1e-5, dtype=dtype, device=torch.device("cpu"))
    with pytest.raises(ValueError, match="pairs"):
        RotaryLatentAttention(64, 2, 8, 5, 8, 16, 1.0, 1e-5, device=torch.device("cpu"))


def test_the_ways_of_a_prompt_step_are_picked_by_its_shape():
    """Short portions behind long histories work in the latents' space, whole prompts of real sizes as heads."""
    from types import SimpleNamespace
    from janus_b200.parts.latent_attention import RotaryLatentAttention
    m = RotaryLatentAttention(2048, 16, 128, 64, 128, 512, 0.07, 1e-5, device=torch.device("cpu"))
    step = lambda q, kv, n=1, decode=False: SimpleNamespace(is_decode=decode, n_tokens=q, kv_total=kv, n_seqs=n)  # noqa: E731
    assert m._as_heads(step(2048, 2048)) and m._as_heads(step(8 * 2048, 8 * 2048, 8)) and m._as_heads(step(1024, 8192))
    assert not m._as_heads(step(2, 2048)) and not m._as_heads(step(16, 65536)) and not m._as_heads(step(8, 8 * 2048, 8, True))


def far_key_case(seed=6):
    """One layer of latent attention alone and two prompts that differ in their first token only.  Those two tokens (and
    no others) have a feature that makes one latent number large; the last token's query asks for it in every head, so
    what the last position says, 400 tokens on, is the first token's value; the two tokens' other features are
    opposite."""
    cfg = config(64, 32, 2.0, [layer(mixer(2, 8, 4, 8, 16, 0.5, 100.0))])
    w = P.random_weights(cfg, seed)
    m, first_a, first_b, last = "l0.mix.", 0, 1, 2
    emb = w["embed"].clone()
    emb[:, 30:] = 0.0
    emb[first_b, :30] = -emb[first_a, :30]
    emb[first_a, 30] = emb[first_b, 30] = emb[last, 31] = 6.0
    w["embed"] = emb
    for name in ("embed.norm.b", "l0.norm1.b"):
        t = w[name].clone()
        t[30:] = 0.0
        w[name] = t
    t = w[m + "dkv"].clone()
    t[:, 30:] = 0.0
    t[0, :30] = 0.0
    t[0, 30] = 6.0
    w[m + "dkv"] = t
    t = w[m + "q"].clone()
    t[:, 30:] = 0.0
    t[[0, 12], 31] = 9.0                       # the first unrotated number of both heads (of 8 + 4 each)
    w[m + "q"] = bf(t)
    t = w[m + "uk"].clone()
    t[[0, 8], 0] = 3.0
    w[m + "uk"] = t
    t = w[m + "uv"].clone()
    t[:, 0] = 0.0                               # the loud number says nothing itself
    w[m + "uv"] = bf(t * 3.0)
    middle = [3 + t % 61 for t in random_tokens(398, 64, seed)]
    return cfg, w, [first_a] + middle + [last], [first_b] + middle + [last]


def test_the_cases_made_to_show_do_show_in_the_plain_logits():
    cfg, w, a, b = far_key_case()
    assert rel_err(plain_logits(cfg, w, a)[-1:], plain_logits(cfg, w, b)[-1:]) > 8 * BF16_TOL
    # an early key that is missed, keys whose positions are off by one, a correction that reaches the weights, a borrowed
    # layer that reads another place's rows: each moves the logits by more than the bounds
    w = weights_for(CFG_A, 12)
    ids = random_tokens(80, CFG_A["vocab"], 5)
    ref = plain_logits(CFG_A, w, ids)
    attend, rotate, choose = P.causal_attention, P.rotate, P.choose_experts

    def changed(cfg=CFG_A, **kw):
        try:
            for k, v in kw.items():
                setattr(P, k, v)
            return P.forward(cfg, w, ids)[0]
        finally:
            P.causal_attention, P.rotate, P.choose_experts = attend, rotate, choose

    def without_the_key_before(q, k, v, start, scale):
        out = attend(q, k, v, start, scale)
        for t in range(1, q.shape[0]):
            keep = [j for j in range(start + t + 1) if j != start + t - 1]
            out[t] = attend(q[t:t + 1], k[keep], v[keep], len(keep) - 1, scale)[0]
        return out

    def corrected_weights(z, c, top, scale):
        chosen, weight = choose(z, c, top, scale)
        return chosen, weight + scale * c[chosen]

    rows = dict(rot_dim=8, kv_rank=24, scale=0.5)
    from_0 = config(160, 64, 2.0, [layer(mixer(2, 8, vdim=16, **rows)), layer(mixer(3, 16, vdim=8, **rows)),
                                   layer(mixer(4, 12, vdim=12, kv_from=0, **rows))])
    from_1 = copy.deepcopy(from_0)
    from_1["layers"][2]["mixer"]["kv_from"] = 1
    w2 = P.random_weights(from_0, 5)
    assert rel_err(P.forward(from_1, w2, ids)[0], P.forward(from_0, w2, ids)[0]) > 1.2 * tol_for("bfloat16")
    for kw in (dict(causal_attention=without_the_key_before), dict(choose_experts=corrected_weights),
               dict(rotate=lambda x, pos, rot: rotate(x, pos + (x.shape[1] == 1), rot))):
        assert rel_err(changed(**kw), ref) > 1.2 * tol_for("bfloat16"), kw


# ------------------------------------------------------------------------------------------------
# on the device: one mechanism at a time
# ------------------------------------------------------------------------------------------------
gpu = pytest.mark.gpu


def load(d, dtype, max_tokens=2048, **kw):
    import janus_b200
    return janus_b200.load(d, dtype=dtype, max_tokens=max_tokens, **kw)


@pytest.fixture(params=["heads", "latents"])
def way(request, monkeypatch):
    """Every prompt step of the bfloat16 engine goes this way through the mixer (where its sizes allow)."""
    from janus_b200.parts.latent_attention import RotaryLatentAttention
    monkeypatch.setattr(RotaryLatentAttention, "prompt_way", request.param)
    return request.param


DTYPES_AND_WAYS = [("float32", "latents"), ("bfloat16", "heads"), ("bfloat16", "latents")]
both = pytest.mark.parametrize("dtype,way", DTYPES_AND_WAYS, indirect=["way"])


@gpu
def test_dynamic_tanh_and_the_sum_around_it_against_the_formula():
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(0)
    for T, W in ((7, 64), (5, 37), (300, 2048), (1, 6)):
        r, y = torch.randn(T, W, generator=g) * 2, torch.randn(T, W, generator=g) * 2
        na = (torch.randn(W, generator=g), torch.randn(W, generator=g), 0.7)
        nb = (torch.randn(W, generator=g), torch.randn(W, generator=g), 1.3)
        cu = lambda n: (n[0].cuda(), n[1].cuda(), n[2])   # noqa: E731
        f = lambda v, n: P.squash(v.to(P.DT), torch.tensor(n[2], dtype=P.DT), n[0].to(P.DT), n[1].to(P.DT))   # noqa: E731
        for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 1e-2)):
            rd, yd = r.cuda(), y.cuda()
            x = torch.empty(T, W, dtype=dtype, device="cuda")
            scratch, scratch2 = torch.ones(64, device="cuda"), torch.ones(400, device="cuda")
            ops.tanh_norm(rd, y=yd, norm_y=cu(na), mult=0.5, norm_x=cu(nb), x_out=x, clear=scratch, clear2=scratch2)
            want = r.to(P.DT) + 0.5 * f(y, na)
            assert rel_err(rd.cpu(), want) < 2e-6 and float(yd.abs().sum()) == 0.0
            assert rel_err(x.float().cpu(), f(want, nb)) < tol
            assert float(scratch.abs().sum()) == 0.0 and float(scratch2.abs().sum()) == 0.0
            # the sum with a cast, the norm alone over picked rows, the stream itself through the norm
            rd, yd = r.cuda(), y.cuda()
            ops.tanh_norm(rd, y=yd, norm_y=cu(na), x_out=x)
            want = r.to(P.DT) + f(y, na)
            assert rel_err(x.float().cpu(), want) < tol
            pick = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)
            x3 = torch.empty(3, W, dtype=dtype, device="cuda")
            rd = r.cuda()
            ops.tanh_norm(rd, norm_x=cu(nb), x_out=x3, row_index=pick.cuda())
            assert rel_err(x3.float().cpu(), f(r[pick.long()], nb)) < tol and torch.equal(rd.cpu(), r)
            ops.tanh_norm(rd, norm_y=cu(na), replace=True)
            assert rel_err(rd.cpu(), f(r, na)) < 2e-6


@gpu
def test_products_with_the_exact_gelu_in_their_epilogue_and_behind_them():
    from types import SimpleNamespace
    from janus_b200.engine.workspace import Workspace
    from janus_b200.kernels import ops
    from janus_b200.parts.feedforward import GeluFeedForward
    g = torch.Generator().manual_seed(2)
    x = torch.linspace(-6.0, 6.0, 4099)
    out = torch.empty(4099, device="cuda")
    ops.activate(x.cuda(), out, "gelu")
    assert float((out.cpu().to(P.DT) - P.gelu(x.to(P.DT))).abs().max()) < 1e-6
    for dtype in (torch.float32, torch.bfloat16):
        for T, W, F in ((3, 64, 200), (70, 96, 136), (300, 256, 512), (20, 36, 50), (9, 256, 20000)):
            h, up, down = (bf(torch.randn(*s, generator=g) * k) for s, k in
                           (((T, W), 1.0), ((F, W), 2.0 * W ** -0.5), ((W, F), F ** -0.5)))
            part = GeluFeedForward(W, F, dtype=dtype)
            part.load(up.to(torch.bfloat16), down.to(torch.bfloat16))
            res = torch.zeros(T, W, device="cuda")
            part.forward(h.to(dtype).cuda(), res, SimpleNamespace(workspace=Workspace(torch.device("cuda"))))
            want = P.dense_ff({"up": up, "down": down}, "", h)
            assert rel_err(res.cpu(), want) < (1e-5 if dtype == torch.float32 else 1.5e-2), (dtype, T, W, F)


def _rotation(r, positions, scaling=None):
    """(table of the library, the plain rotation) for vectors of r numbers."""
    from janus_b200.parts.base import PartSpec, make_part
    if r == 0:
        return None, lambda x: x
    rot = dict(dims=r, base=300.0)
    if scaling:
        rot["scaling"] = scaling
    table = make_part("position", PartSpec("ramped_rotary", dict(dims=r, theta=300.0, max_positions=1024, scaling=scaling)),
                      torch.float32, torch.device("cuda")).fused_rotary_table()
    return table, lambda x: P.rotate(x, positions, rot)


@gpu
@pytest.mark.parametrize("H,d,r,e,n", [(4, 16, 8, 24, 40), (3, 5, 6, 7, 11), (2, 128, 64, 128, 512), (1, 8, 2, 1, 8), (5, 3, 0, 6, 13),
                                       (16, 64, 32, 64, 256)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_queries_rows_and_values_of_latent_attention_against_the_plain_steps(H, d, r, e, n, dtype):
    """Queries as heads and in the latents' space, the token's row in its page (and its copy), rows gathered back from
    pages out of order, values from rows and from the partial sums of key splits, with and without the gate."""
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    T, PAGE, eps = 11, 64, 1e-5
    stored = (n + r + 7) // 8 * 8 if dtype == torch.bfloat16 else n + r
    dp = (d + r + 7) // 8 * 8
    tol = 3e-6 if dtype == torch.float32 else 1e-2
    positions = torch.tensor([0, 1, 5, 6, 7, 62, 63, 64, 700, 701, 1023])
    table, turn = _rotation(r, positions, dict(factor=4.0, original=100, fast=8.0, slow=1.0))
    qw = H * (d + r)
    proj = torch.randn(T, qw + H * e + n + r, generator=g)
    col = qw + H * e
    q = proj[:, :qw].to(P.DT).view(T, H, d + r)
    turned = turn(q[..., d:])
    weight = torch.randn(n, generator=g)
    c = P.rms_unit(proj[:, col:col + n].to(P.DT), eps) * weight.to(P.DT)
    part = turn(proj[:, None, col + n:].to(P.DT))[:, 0]
    want_row = torch.cat([c, part], dim=-1)
    uk, uv = bf(torch.randn(H * d, n, generator=g) * n ** -0.5), bf(torch.randn(H * e, n, generator=g) * n ** -0.5)
    dest = torch.tensor([3 * PAGE + 63, 0, 1, 2, PAGE + 7, 5, 2 * PAGE, 63, 64, 70, 100], dtype=torch.int32)
    for kind in ("heads", "latents"):
        pages = torch.zeros(4, 1, PAGE, stored, dtype=dtype, device="cuda")
        rows = torch.full((T, stored), 7.0, dtype=dtype, device="cuda")
        row = (col, n, stored, weight.cuda(), eps, dest.cuda(), pages)
        if kind == "heads":
            out = torch.empty(T, H * dp, dtype=dtype, device="cuda")
            ops.latent_heads(proj.cuda(), 0, H, d, r, dp, table, positions.int().cuda(), out, row, rows)
            want = torch.cat([q[..., :d], turned, torch.zeros(T, H, dp - d - r, dtype=P.DT)], dim=-1)
            assert rel_err(rows[:, :n + r].float().cpu(), want_row) < tol and float(rows[:, n + r:].abs().sum()) == 0.0
        else:
            out = torch.empty(T, H * stored, dtype=dtype, device="cuda")
            ops.latent_queries(proj.cuda(), 0, H, d, r, n, stored, uk.to(dtype).cuda(), table, positions.int().cuda(), out, row)
            want = torch.cat([torch.einsum("thd,hdn->thn", q[..., :d], uk.view(H, d, n)), turned,
                              torch.zeros(T, H, stored - n - r, dtype=P.DT)], dim=-1)
        assert rel_err(out.float().cpu().view(want.shape), want) < tol, kind
        flat = pages.view(-1, stored).float().cpu()
        assert rel_err(flat[dest.long(), :n + r], want_row) < tol, kind
        others = [i for i in range(4 * PAGE) if i not in dest.tolist()]
        assert float(flat[others].abs().sum()) == 0.0 and float(flat[:, n + r:].abs().sum()) == 0.0
        # the queries alone (a place that reads another place's rows): the pages stay as they are
        before, out2 = pages.clone(), torch.empty_like(out)
        if kind == "heads":
            ops.latent_heads(proj.cuda(), 0, H, d, r, dp, table, positions.int().cuda(), out2)
        else:
            ops.latent_queries(proj.cuda(), 0, H, d, r, n, stored, uk.to(dtype).cuda(), table, positions.int().cuda(), out2)
        assert torch.equal(out, out2) and torch.equal(before, pages)
    o = bf(torch.randn(T, H, n, generator=g))
    gate_cols = proj[:, qw:col].to(P.DT)
    ep = (e + 7) // 8 * 8
    plain = torch.einsum("thn,hen->the", o, uv.view(H, e, n))
    for gated in (True, False):
        out = torch.full((T, H * ep), 9.0, dtype=dtype, device="cuda")
        gate = proj.cuda()[:, qw:col] if gated else None
        ops.latent_values(o.to(dtype).cuda().view(T, H * n), None, uv.to(dtype).cuda(), gate, out, H, n, e, ep)
        want = plain * torch.sigmoid(gate_cols).view(T, H, e) if gated else plain
        got = out.view(T, H, ep).float().cpu()
        assert rel_err(got[..., :e], want) < tol and float(got[..., e:].abs().sum()) == 0.0
    # partial sums of three splits, one of them without keys: o = sum_s 2^(m_s) part_s / sum_s 2^(m_s) l_s
    sums = torch.randn(T, H, 3, n, generator=g)
    m, l = torch.randn(T, H, 3, generator=g) * 3, torch.rand(T, H, 3, generator=g) + 0.5
    sums[:, :, 1], m[:, :, 1], l[:, :, 1] = 0.0, -math.inf, 0.0
    f = torch.exp2(m.to(P.DT))
    joined = (f[..., None] * sums.to(P.DT)).sum(2) / (f * l.to(P.DT)).sum(2)[..., None]
    out = torch.empty((T, H * ep), dtype=dtype, device="cuda")
    ops.latent_values(None, (sums.cuda(), torch.stack([m, l], dim=-1).contiguous().cuda(), 3), uv.to(dtype).cuda(), None, out,
                      H, n, e, ep)
    assert rel_err(out.view(T, H, ep).float().cpu()[..., :e], torch.einsum("thn,hen->the", joined, uv.view(H, e, n))) < tol
    if dtype == torch.bfloat16:
        cache = torch.randn(7, 1, PAGE, stored, generator=g).to(dtype)
        lens, order = [70, 1, 128, 0], [[5, 2], [6], [0, 3], []]
        bt = torch.full((4, 3), -1, dtype=torch.int32)
        for s, ps in enumerate(order):
            bt[s, :len(ps)] = torch.tensor(ps, dtype=torch.int32)
        start = torch.tensor([0, 70, 71, 199, 199], dtype=torch.int32)
        got = torch.empty(199, stored, dtype=dtype, device="cuda")
        ops.gather_rows(cache.cuda(), bt.cuda(), torch.tensor(lens, dtype=torch.int32).cuda(), start.cuda(), got, PAGE, 4)
        want = torch.cat([cache[ps].reshape(-1, stored)[:n_] for ps, n_ in zip(order, lens) if n_])
        assert torch.equal(got.cpu(), want)


def _paged_rows(rows, order, n_pages):
    """Pages that hold the given sequences' rows ([len, stored] each), pages handed out in `order`; (pages, block table)."""
    PAGE = 64
    stored = rows[0].shape[1]
    pages = torch.zeros(n_pages, 1, PAGE, stored, dtype=torch.float64)
    width = max((len(x) + PAGE - 1) // PAGE for x in rows) + 1
    table = torch.full((len(rows), width), -1, dtype=torch.int32)
    it = iter(order)
    for s, x in enumerate(rows):
        for i in range((len(x) + PAGE - 1) // PAGE):
            p = next(it)
            table[s, i] = p
            piece = x[i * PAGE:(i + 1) * PAGE]
            pages[p, 0, :len(piece)] = piece
    return pages, table


def _latent_attention_want(q, rows, n, lens, q_lens, scale):
    out, at = [], 0
    for x, ql in zip(rows, q_lens):
        k = x[:, None, :].expand(len(x), q.shape[1], x.shape[1])
        out.append(P.causal_attention(q[at:at + ql], k, k[..., :n], len(x) - ql, scale))
        at += ql
    return torch.cat(out)


@gpu
@pytest.mark.parametrize("H,n,r", [(4, 40, 8), (3, 11, 6), (16, 256, 64), (20, 264, 64), (33, 24, 2), (1, 1016, 64)])
@pytest.mark.parametrize("splits", [None, 1, 2, 5])
def test_attention_over_cached_rows_against_the_plain_softmax(H, n, r, splits):
    """Single tokens and portions of unequal sequences in one launch, one to many pages, whole and in key splits (some
    without keys); every query has one loud key, at its own position, at the first one, or next to a page's edge."""
    from janus_b200.engine.workspace import Workspace
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    stored = (n + r + 7) // 8 * 8
    for lens, q_lens in (([1, 64, 65, 700, 33], [1] * 5), ([1, 70, 129, 400], [1, 5, 66, 2])):
        rows = []
        for L in lens:
            x = torch.zeros(L, stored, dtype=P.DT)
            x[:, :n + r] = bf(torch.randn(L, n + r, generator=g))
            rows.append(x)
        T = sum(q_lens)
        q = torch.zeros(T, H, stored, dtype=P.DT)
        q[..., :n + r] = bf(torch.randn(T, H, n + r, generator=g))
        at = 0
        for x, ql in zip(rows, q_lens):
            for i in range(ql):
                pos = len(x) - ql + i
                for h in range(H):
                    loud = [pos, 0, min(pos, 63), min(pos, 64), max(0, pos - 1)][(i + h) % 5]
                    q[at + i, h] = bf(q[at + i, h] * 0.3 + 1.5 * x[loud])
            at += ql
        scale = 6.0 / (n + r)
        pages, table = _paged_rows(rows, torch.randperm(40, generator=g).tolist(), 40)
        kv_len = torch.tensor(lens, dtype=torch.int32).cuda()
        q_start = torch.tensor([0] + list(np.cumsum(q_lens)), dtype=torch.int32).cuda()
        ws = Workspace(torch.device("cuda"))
        out = torch.empty(T, H * n, dtype=torch.bfloat16, device="cuda")
        partial = ops.latent_attention(q.to(torch.bfloat16).cuda().view(T, -1), pages.to(torch.bfloat16).cuda(), out, table.cuda(),
                                       q_start, kv_len, len(lens), max(q_lens), H, stored, n, 64, scale, ws, max(lens),
                                       n_splits=splits)
        if partial is not None:
            so, ml, k = partial
            so, ml = so.cpu().to(P.DT).view(T, H, k, n), ml.cpu().to(P.DT).view(T, H, k, 2)
            f = torch.exp2(ml[..., 0] - ml[..., 0].max(dim=-1, keepdim=True).values)
            got = (so * f[..., None]).sum(2) / (f * ml[..., 1]).sum(2)[..., None]
        else:
            got = out.float().cpu().view(T, H, n)
        want = _latent_attention_want(q, rows, n, lens, q_lens, scale)
        assert rel_err(got, want) < 1.5e-2, (lens, splits)
        # the float32 kernel on the same case
        seq = torch.tensor([s for s, k in enumerate(q_lens) for _ in range(k)], dtype=torch.int32).cuda()
        pos = torch.tensor([L - k + i for L, k in zip(lens, q_lens) for i in range(k)], dtype=torch.int32).cuda()
        if splits is None:
            p32 = pages.float().cuda()
            out32 = torch.empty(T, H * n, device="cuda")
            ops.attention_f32(q.float().cuda().view(T, -1), p32, p32, out32, table.cuda(), seq, pos, H, 1, stored, 64, 0, scale, vd=n)
            assert rel_err(out32.cpu().view(T, H, n), want) < 1e-5


@gpu
@pytest.mark.parametrize("tiles", ["1", "2"])
@pytest.mark.parametrize("H,hd,vd", [(4, 16, 8), (3, 96, 64), (2, 192, 128), (5, 128, 128), (2, 136, 16), (2, 256, 248), (6, 72, 72)])
def test_attention_over_a_matrix_of_keys_and_values_against_the_plain_softmax(H, hd, vd, tiles, monkeypatch):
    """Whole prompts and portions of unequal sequences that lie one after another in the matrix; every query has one
    loud key at an edge of a page, of a block or of the sequence."""
    from janus_b200.kernels import ops
    monkeypatch.setenv("JANUS_ATTN_TC_TILES", tiles)
    g = torch.Generator().manual_seed(5)
    for lens, q_lens in (([1, 64, 200, 129], [1, 64, 200, 129]), ([70, 333, 65], [3, 130, 1])):
        L, T = sum(lens), sum(q_lens)
        kv = bf(torch.randn(L, H * (hd + vd), generator=g))
        k, v = kv[:, :H * hd].view(L, H, hd), kv[:, H * hd:].view(L, H, vd)
        q = bf(torch.randn(T, H, hd, generator=g) * 0.3)
        starts, at = [0] + list(np.cumsum(lens)), 0
        for s, (n, ql) in enumerate(zip(lens, q_lens)):
            for i in range(ql):
                pos = n - ql + i
                for h in range(H):
                    loud = [pos, 0, min(pos, 63), min(pos, 64), min(pos, 127), min(pos, 128)][(i + h) % 6]
                    q[at + i, h] = bf(q[at + i, h] + 1.5 * k[starts[s] + loud, h])
            at += ql
        scale = 6.0 / hd
        out = torch.empty(T, H * vd, dtype=torch.bfloat16, device="cuda")
        i32 = lambda x: torch.tensor(x, dtype=torch.int32).cuda()      # noqa: E731
        ops.attention_tc_matrix(q.to(torch.bfloat16).cuda().view(T, -1), kv.to(torch.bfloat16).cuda(), out, i32(starts),
                                i32([0] + list(np.cumsum(q_lens))), i32(lens), len(lens), max(q_lens), H, hd, vd, max(lens), scale)
        ops.check_kernel_status(torch.device("cuda"))
        got, at = out.float().cpu().view(T, H, vd), 0
        for s, (n, ql) in enumerate(zip(lens, q_lens)):
            want = P.causal_attention(q[at:at + ql], k[starts[s]:starts[s] + n], v[starts[s]:starts[s] + n], n - ql, scale)
            assert rel_err(got[at:at + ql], want) < 1.5e-2, (lens, s)
            at += ql


@gpu
def test_router_with_corrected_choice_and_scaled_weights():
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(6)
    for T, E, top, scale in ((9, 6, 2, 1.7), (70, 64, 6, 0.5), (1, 1, 1, 1.0), (5, 40, 16, 2.5), (33, 5, 5, 1.0)):
        z = torch.randn(T, E, generator=g) * 2
        corr = torch.randn(E, generator=g) * 0.6 - 0.8
        wide = torch.cat([z, torch.full((T, 1), 99.0)], dim=1)
        se, sw = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
        ops.route_topk(wide.cuda(), top, se, sw, experts=E, correction=corr.cuda(), scale=scale)
        chosen, weight = P.choose_experts(z.to(P.DT), corr.to(P.DT), top, scale)
        assert torch.equal(se.cpu().long(), chosen), (T, E)
        assert rel_err(sw.cpu(), weight) < 1e-5
    # equal corrections change nothing but are no part of the weights; the lower index wins a tie
    z = torch.tensor([[0.3, 0.3, -1.0, 0.3]])
    se, sw = torch.empty(1, 2, dtype=torch.int32, device="cuda"), torch.empty(1, 2, device="cuda")
    ops.route_topk(z.cuda(), 2, se, sw, correction=torch.full((4,), 5.0).cuda())
    assert se.tolist() == [[0, 1]] and rel_err(sw.cpu(), torch.sigmoid(z[:, :2].to(P.DT))) < 1e-6


@gpu
@pytest.mark.parametrize("on_output", [True, False])
@pytest.mark.parametrize("T,W,F,E,top", [(3, 64, 96, 6, 2), (1, 32, 32, 3, 3), (40, 128, 160, 2, 1), (150, 96, 64, 5, 3),
                                         (8, 2048, 1440, 4, 2)])
def test_experts_of_few_pairs_on_the_tensor_cores_against_the_formula(T, W, F, E, top, on_output):
    """Few and many pairs per expert (more than one launch group of 32 and one list of 256), experts that nobody chose,
    the weight on the output and on the input; the results are added to what is there."""
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(8)
    h = bf(torch.randn(T, W, generator=g))
    m = {k: bf(torch.randn(*shape, generator=g) * shape[-1] ** -0.5) for k, shape in
         (("gate", (E, F, W)), ("up", (E, F, W)), ("down", (E, W, F)))}
    pick = torch.stack([torch.randperm(max(E - 1, top), generator=g)[:top] for _ in range(T)])      # the last expert idles
    weight = torch.rand(T, top, generator=g) + 0.2
    out = torch.randn(T, W, generator=g)
    want = out.to(P.DT)
    for t in range(T):
        for j in range(top):
            e = int(pick[t, j])
            x = h[t] if on_output else bf(h[t] * weight[t, j])
            y = m["down"][e] @ bf(P.silu(m["gate"][e] @ x) * (m["up"][e] @ x))
            want[t] += y * weight[t, j].to(P.DT) if on_output else y
    cu = lambda t: t.to(torch.bfloat16).cuda()       # noqa: E731
    got, act = out.cuda(), torch.empty(T * top, F, dtype=torch.bfloat16, device="cuda")
    ops.experts_few_tokens_tc(cu(h), pick.int().cuda(), weight.cuda(), cu(m["gate"]), cu(m["up"]), cu(m["down"]), act, got,
                              weight_on_output=on_output)
    assert rel_err(got.cpu(), want) < 4e-3


# ------------------------------------------------------------------------------------------------
# on the device: the engine
# ------------------------------------------------------------------------------------------------
@gpu
@both
@pytest.mark.parametrize("name,which", [("A", 0), ("A", 1), ("C", 0), ("C", 2), ("D", 1)])
def test_the_mixer_alone_in_a_layer_without_feed_forward(tmp_path, name, which, dtype, way):
    from janus_b200.engine import StepEntry
    cfg = dict(CONFIGS[name], layers=[dict(CONFIGS[name]["layers"][which], mlp=None)])
    d, w = folder(tmp_path, cfg, 20 + which)
    model = load(d, dtype, max_tokens=512, max_slots=2)
    ids = random_tokens(150, cfg["vocab"], which)
    slot = model.alloc_slot()
    out = [model.step([StepEntry(slot, ids[:100], range(100))]).cpu(), model.step([StepEntry(slot, ids[100:140], range(40))]).cpu()]
    out += [model.step([StepEntry(slot, [t], [0])]).cpu() for t in ids[140:]]
    assert rel_err(torch.cat(out), plain_logits(cfg, w, ids)) < tol_for(dtype)
    model.check()


@gpu
@both
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_prompts_of_unequal_lengths_in_one_step(tmp_path, name, dtype, way):
    from janus_b200.engine import StepEntry
    cfg = CONFIGS[name]
    d, w = folder(tmp_path, cfg, 11)
    model = load(d, dtype, max_tokens=64 * 16, max_slots=4)
    seqs = [random_tokens(n, cfg["vocab"], n) for n in (1, 64, 330, 129)]
    slots = [model.alloc_slot() for _ in seqs]
    out = model.step([StepEntry(s, ids, range(len(ids))) for s, ids in zip(slots, seqs)]).cpu()
    row = 0
    for ids in seqs:
        assert rel_err(out[row:row + len(ids)], plain_logits(cfg, w, ids)) < tol_for(dtype), len(ids)
        row += len(ids)
    model.check()


@gpu
@both
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_then_single_tokens_in_a_batch_and_slots_used_again(tmp_path, name, dtype, way):
    """Prompts cut into portions of 2 to 64 tokens, unequal requests in one batch, then one token each until the
    shorter ones have ended; afterwards other requests take the freed slots and pages.  Every row is compared with the
    whole sequence's plain logits."""
    from janus_b200.engine import StepEntry
    cfg = CONFIGS[name]
    d, w = folder(tmp_path, cfg, 12)
    model = load(d, dtype, max_tokens=64 * 9, max_slots=3)
    for round_no, lengths in enumerate(((140, 75, 20), (90, 130, 129))):
        seqs = [random_tokens(n, cfg["vocab"], 7 * round_no + n) for n in lengths]
        ref = [plain_logits(cfg, w, ids) for ids in seqs]
        got = [[] for _ in seqs]
        slots = [model.alloc_slot() for _ in seqs]
        at = [0, 0, 0]
        for portion in ((2, 3, 2), (62, 5, 3), (1, 40, 2), (17, 2, 2)):
            entries = []
            for i, n in enumerate(portion):
                entries.append(StepEntry(slots[i], seqs[i][at[i]:at[i] + n], range(n)))
                at[i] += n
            out = model.step(entries).cpu()
            row = 0
            for i, n in enumerate(portion):
                got[i].append(out[row:row + n])
                row += n
        live = [0, 1, 2]
        while live:
            out = model.step([StepEntry(slots[i], [seqs[i][at[i]]], [0]) for i in live]).cpu()
            for row, i in enumerate(live):
                got[i].append(out[row:row + 1])
                at[i] += 1
            for i in [i for i in live if at[i] == len(seqs[i])]:
                model.free_slot(slots[i])
                live.remove(i)
        for i in range(3):
            assert rel_err(torch.cat(got[i]), ref[i]) < tol_for(dtype), (round_no, i)
        model.engine.cache.check()
    model.check()


def drawn_config(seed):
    """A configuration drawn from a seed: two to five layers, feed-forward or none, sizes that are multiples of nothing
    as often as not, layers that borrow an earlier layer's rows now and then."""
    r = np.random.RandomState(seed)
    pick = lambda *xs: xs[r.randint(len(xs))]  # noqa: E731
    layers = []
    for i in range(r.randint(2, 6)):
        heads, d, e = int(pick(1, 2, 3, 4, 5, 8)), int(pick(4, 8, 10, 16, 24, 40)), int(pick(4, 8, 9, 16, 24, 32))
        scale = float(pick(0.3, 0.5, 0.8)) * 8 ** -0.5
        own = [j for j, x in enumerate(layers) if "kv_from" not in x["mixer"]]
        if own and r.rand() < 0.35:
            j = int(pick(*own))
            m = layers[j]["mixer"]
            mx = dict(m, heads=heads, dim=d, vdim=e, scale=scale, kv_from=j)
        else:
            n, rot = [(40, 8), (11, 6), (24, 2), (8, 8)][r.randint(4)]
            mx = mixer(heads, d, rot, e, n, scale, float(pick(50.0, 10000.0)), pick(None, _YARN, (2.0, 300, 16.0, 2.0)))
        kind = r.randint(4)
        if kind == 0:
            mlp = None
        elif kind == 1:
            mlp = dense(int(pick(24, 40, 64, 100)))
        else:
            E = int(pick(1, 2, 3, 5, 8))
            mlp = moe(int(pick(16, 24, 33, 64)), E, 1 + r.randint(min(E, 4)), float(pick(0.7, 1.0, 2.3)))
        layers.append(layer(mx, mlp))
    return config(int(pick(50, 97, 128)), int(pick(32, 40, 64, 72, 36, 128)), float(pick(1.0, 4.0, 8.5)), layers,
                  eps=float(pick(1e-5, 1e-6)))


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(1, 17)))
def test_configurations_drawn_from_a_seed(tmp_path, seed, dtype):
    """Whatever the sizes, the order of the layers and the options: a prompt, a portion, single tokens and a second
    request beside them give the plain logits."""
    from janus_b200.engine import StepEntry
    cfg = drawn_config(seed)
    d, w = folder(tmp_path, cfg, 100 + seed)
    model = load(d, dtype, max_tokens=64 * 8, max_slots=2)
    a, b = random_tokens(150, cfg["vocab"], seed), random_tokens(40, cfg["vocab"], seed + 50)
    ra, rb = plain_logits(cfg, w, a), plain_logits(cfg, w, b)
    sa, sb = model.alloc_slot(), model.alloc_slot()
    out = model.step([StepEntry(sa, a[:70], range(70)), StepEntry(sb, b[:33], [0, 32])]).cpu()
    ga, gb = [out[:70]], [out[70:]]
    ga.append(model.step([StepEntry(sa, a[70:143], range(73))]).cpu())
    for j in range(7):
        out = model.step([StepEntry(sa, [a[143 + j]], [0]), StepEntry(sb, [b[33 + j]], [0])]).cpu()
        ga.append(out[:1])
        gb.append(out[1:])
    text = json.dumps(cfg)
    assert rel_err(torch.cat(ga), ra) < tol_for(dtype), text
    assert rel_err(torch.cat(gb), rb[[0, 32, *range(33, 40)]]) < tol_for(dtype), text
    model.check()


@gpu
@both
def test_a_batch_gives_every_request_what_it_gets_alone(tmp_path, dtype, way):
    """The engine against itself: four unequal requests in one batch (prompt, then single tokens) and each alone, on
    slots and pages that other requests held before; rows differ by rounding at most."""
    from janus_b200.engine import StepEntry
    cfg = CFG_A
    d, _ = folder(tmp_path, cfg, 13)
    model = load(d, dtype, max_tokens=64 * 12, max_slots=4)
    seqs = [random_tokens(n, cfg["vocab"], 50 + n) for n in (100, 3, 65, 31)]
    alone = []
    for ids in seqs:
        slot = model.alloc_slot()
        rows = [model.step([StepEntry(slot, ids[:-2], [len(ids) - 3])]).cpu()]
        rows += [model.step([StepEntry(slot, [t], [0])]).cpu() for t in ids[-2:]]
        alone.append(torch.cat(rows))
        model.free_slot(slot)
    slots = [model.alloc_slot() for _ in seqs]
    first = model.step([StepEntry(s, ids[:-2], [len(ids) - 3]) for s, ids in zip(slots, seqs)]).cpu()
    tails = [model.step([StepEntry(s, [ids[len(ids) - 2 + j]], [0]) for s, ids in zip(slots, seqs)]).cpu() for j in range(2)]
    slack = 1e-5 if dtype == "float32" else BF16_TOL
    for i in range(4):
        assert rel_err(torch.stack([first[i], tails[0][i], tails[1][i]]), alone[i]) < slack, i
    model.check()


@gpu
@both
def test_a_far_key_is_found_in_prompts_portions_and_single_tokens(tmp_path, dtype, way):
    from janus_b200.engine import StepEntry
    cfg, w, a, b = far_key_case()
    d = P.save_folder(cfg, w, str(tmp_path / "far"))
    model = load(d, dtype, max_tokens=1024, max_slots=2)
    tol = 5 * FP32_TOL if dtype == "float32" else tol_for(dtype)
    for ids in (a, b):
        ref = plain_logits(cfg, w, ids)[-1:]
        for cuts in ([400], [1, 397, 2], [64, 64, 64, 64, 64, 78, 2], [398, 1, 1], [399, 1], [63, 2, 335]):
            slot, at = model.alloc_slot(), 0
            for n in cuts:
                last = at + n == 400
                out = model.step([StepEntry(slot, ids[at:at + n], [n - 1] if last else [])])
                at += n
            assert at == 400 and rel_err(out.cpu(), ref) < tol, cuts
            model.free_slot(slot)
    model.check()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_from_the_first_token(tmp_path, name, dtype):
    """200 single tokens from position 0 on (pages fill and new ones are taken), two sequences a step, one of them a few
    tokens behind."""
    from janus_b200.engine import StepEntry
    cfg = CONFIGS[name]
    d, w = folder(tmp_path, cfg, 17)
    model = load(d, dtype, max_tokens=64 * 8, max_slots=2)
    a, b = random_tokens(200, cfg["vocab"], 1), random_tokens(195, cfg["vocab"], 2)
    sa, sb = model.alloc_slot(), model.alloc_slot()
    ga, gb = [], []
    for t in range(200):
        entries = [StepEntry(sa, [a[t]], [0])] + ([StepEntry(sb, [b[t - 5]], [0])] if t >= 5 else [])
        out = model.step(entries).cpu()
        ga.append(out[:1])
        if t >= 5:
            gb.append(out[1:])
    assert rel_err(torch.cat(ga), plain_logits(cfg, w, a)) < tol_for(dtype)
    assert rel_err(torch.cat(gb), plain_logits(cfg, w, b)) < tol_for(dtype)
    model.check()


@gpu
@both
def test_a_long_prompt_in_one_step_and_in_portions(tmp_path, dtype, way):
    """700 tokens over eleven pages; then the same prompt in portions of 300, 257 and 143 tokens on a slot that was used
    before, beside a second request."""
    from janus_b200.engine import StepEntry
    cfg = CFG_D
    d, w = folder(tmp_path, cfg, 19)
    model = load(d, dtype, max_tokens=64 * 24, max_slots=2)
    ids, other = random_tokens(700, cfg["vocab"], 9), random_tokens(90, cfg["vocab"], 10)
    ref, ref2 = plain_logits(cfg, w, ids), plain_logits(cfg, w, other)
    want = list(range(0, 700, 7)) + [699]
    slot = model.alloc_slot()
    out = model.step([StepEntry(slot, ids, want)]).cpu()
    assert rel_err(out, ref[want]) < tol_for(dtype)
    model.free_slot(slot)
    slot, second = model.alloc_slot(), model.alloc_slot()
    at, rows = 0, []
    for n, m in ((300, 30), (257, 30), (143, 30)):
        mine = [w_ - at for w_ in want if at <= w_ < at + n]
        b0 = 30 * len(rows)
        out = model.step([StepEntry(second, other[b0:b0 + m], range(m)), StepEntry(slot, ids[at:at + n], mine)]).cpu()
        assert rel_err(out[:m], ref2[b0:b0 + m]) < tol_for(dtype)
        rows.append(out[m:])
        at += n
    assert rel_err(torch.cat(rows), ref[want]) < tol_for(dtype)
    model.check()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point_and_the_scheduler(tmp_path, dtype):
    """`load` -> `generate`: five prompts in batches of two; every generated token is the plain implementation's
    pick given the tokens before it.  A folder made by `write_random_model` loads and generates too."""
    import janus_b200
    from janus_b200.weights import write_random_model
    d, w = folder(tmp_path, CFG_A, 31)
    model = janus_b200.load(d, dtype=dtype, max_tokens=1024, max_slots=4)
    prompts = [random_tokens(n, CFG_A["vocab"], 3 + n) for n in (5, 70, 1, 33, 12)]
    out, stats = model.generate(prompts, max_tokens=10, batch_size=2)
    assert stats.batches == 3
    for p, o in zip(prompts, out):
        assert len(o) == 10
        logits = plain_logits(CFG_A, w, list(p) + list(o))
        for j, tok in enumerate(o):
            row = logits[len(p) - 1 + j]
            slack = 1e-4 if dtype == "float32" else BF16_TOL
            assert float(row.max() - row[tok]) <= slack * float(row.abs().max()), (p, j)
    d2 = write_random_model(CFG_B, str(tmp_path / "gen"), seed=32, dtype="bfloat16", std=0.1, norm_std=0.05)
    cfg2, w2 = P.read_folder(d2)
    assert cfg2["layers"][2]["mlp"]["router"]["experts"] == 4 and set(w2) == set(P.random_weights(CFG_B, 0))
    model = janus_b200.load(d2, dtype=dtype, max_tokens=512, max_slots=2)
    out, _ = model.generate([[1, 2, 3], [4]], max_tokens=6, batch_size=2)
    assert [len(o) for o in out] == [6, 6] and all(0 <= t < CFG_B["vocab"] for o in out for t in o)


@gpu
def test_the_replay_program_serves_the_design(tmp_path):
    d, w = folder(tmp_path, CFG_C, 14)
    cfg = CFG_C
    ids, other = random_tokens(40, cfg["vocab"], 2), random_tokens(33, cfg["vocab"], 3)
    steps = [dict(step=0, entries=[dict(id="x", tokens=ids[:30], want=[0, 29]), dict(id="y", tokens=other[:31], want=[30])],
                  end=[])]
    for j in range(10):
        entries = [dict(id="x", tokens=[ids[30 + j]], want=[0])]
        if j < 2:
            entries.append(dict(id="y", tokens=[other[31 + j]], want=[0]))
        steps.append(dict(step=j + 1, entries=entries, end=(["y"] if j == 1 else []) + (["x"] if j == 9 else [])))
    rx, ry = plain_logits(cfg, w, ids), plain_logits(cfg, w, other)
    want = [rx[0], rx[29], ry[30], rx[30], ry[31], rx[31], ry[32]] + [rx[t] for t in range(32, 40)]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype,
                              "--out", str(out), "--max-tokens", "128"],
                             input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
        assert res.returncode == 0, res.stderr[-2000:]
        got = np.concatenate([np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for s in steps])
        assert rel_err(got, torch.stack(want)) < tol_for(dtype)


@gpu
def test_the_command_line_samples_from_the_design(tmp_path):
    """`python -m janus_b200 DIR ...`: greedy tokens are the plain implementation's picks, and sampling with a
    temperature, top-k and a seed runs through the device sampler; a folder with config.json alone runs with
    `--random-weights`."""
    d, w = folder(tmp_path, CFG_D, 15)
    base = [sys.executable, "-m", "janus_b200", d, "3,1,4,1,5", "9,2,6", "--max-tokens", "7", "--dtype", "float32", "--json"]
    env = dict(os.environ, PYTHONPATH=os.pathsep.join([ROOT, os.environ.get("PYTHONPATH", "")]))
    res = subprocess.run(base, capture_output=True, text=True, timeout=900, env=env)
    assert res.returncode == 0, res.stderr[-2000:]
    greedy = json.loads(res.stdout.strip().splitlines()[-1])["tokens"]
    for p, o in zip(([3, 1, 4, 1, 5], [9, 2, 6]), greedy):
        assert len(o) == 7
        logits = plain_logits(CFG_D, w, p + o)
        assert all(int(logits[len(p) - 1 + j].argmax()) == tok for j, tok in enumerate(o))
    res = subprocess.run(base + ["--temperature", "0.9", "--top-k", "12", "--top-p", "0.9", "--seed", "4"],
                         capture_output=True, text=True, timeout=900, env=env)
    assert res.returncode == 0, res.stderr[-2000:]
    sampled = json.loads(res.stdout.strip().splitlines()[-1])["tokens"]
    assert [len(o) for o in sampled] == [7, 7] and all(0 <= t < CFG_D["vocab"] for o in sampled for t in o)
    only_config = tmp_path / "only_config"
    only_config.mkdir()
    (only_config / "config.json").write_text(json.dumps(CFG_A))
    res = subprocess.run([sys.executable, "-m", "janus_b200", str(only_config), "1,2,3", "--max-tokens", "4", "--random-weights",
                          "--json"], capture_output=True, text=True, timeout=900, env=env)
    assert res.returncode == 0, res.stderr[-2000:]
    assert len(json.loads(res.stdout.strip().splitlines()[-1])["tokens"][0]) == 4
