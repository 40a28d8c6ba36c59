"""The Mibezen design in the library against the plain implementation of `plain_mibezen.py`: small configurations made
here (sizes and options that differ from each other in every respect), random weights, every comparison on logits or on
one mechanism's output.  CPU tests cover the plain implementation itself, the configuration reader, the model description
and the cache's chunks; GPU tests cover the kernels one mechanism at a time and the engine: prompts, portions, single
tokens, unequal batches, slots and pages used again, far keys, the edges of chunks and pages, the first tokens, long
decoding, generation.  Prompt steps of the bfloat16 engine have two ways through latent attention (as heads, in the
latents' space); both are held to every case."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_mibezen as P
from helpers import BF16_TOL, FP32_TOL, ROOT, random_tokens, rel_err


def tol_for(dtype):
    """The float32 engine is held to the library's float32 bound.  In bfloat16 the models here are 32 to 128 wide with
    peaked attention: twice the library's bound (a key seen or missed by mistake moves these logits by far more; the cases
    below show it)."""
    return FP32_TOL if dtype == "float32" else 2 * BF16_TOL


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=1000.0, scaling=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale)
    if rot_dim:
        m["rot"] = dict(dims=rot_dim, base=base)
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return m


def chunked(heads, kv_heads, dim, vdim, scale, size, v_mix=False):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size) if size else None,
                v_mix=v_mix)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def layer(mix, mlp=None):
    return dict(type="latent_attention" if "kv_rank" in mix else "attention", mixer=mix, mlp=mlp)


def config(vocab, width, layers, cap=20.0, eps=1e-5):
    return dict(architecture="Mibezen", vocab=vocab, width=width, norm=dict(eps=eps), logit_softcap=cap, layers=layers)


_YARN = (4.0, 64, 8.0, 1.0)
# chunks of several sizes in one model, three layers that mix values around one that does not, values smaller and larger
# than keys, latent layers with and without scaled rotation; experts, dense and none
CFG_A = config(160, 64, [
    layer(chunked(4, 2, 16, 8, 0.3, 50, True), dense(96)),
    layer(latent(4, 16, 8, 24, 20, 40, 0.25, 1000.0, _YARN), moe(48, 6, 2)),
    layer(chunked(6, 3, 24, 8, 0.2, 37), None),
    layer(chunked(2, 2, 8, 8, 0.5, 128, True), moe(32, 5, 3)),
    layer(latent(3, 8, 4, 8, 12, 24, 0.3, 50.0), dense(40)),
    layer(chunked(8, 2, 16, 8, 0.3, 64, True), dense(64))], cap=8.0)
# values that happen to be 1 or equal: one head, all sizes the same, one expert of one, scales of 1, chunks of one token,
# chunks of a page, no cap
CFG_B = config(200, 96, [
    layer(latent(1, 8, 8, 8, 8, 8, 0.4, 50.0), moe(40, 1, 1)),
    layer(chunked(1, 1, 8, 8, 1.0, 1, True), dense(8)),
    layer(chunked(8, 1, 8, 8, 0.5, 64, True), moe(64, 4, 1)),
    layer(latent(2, 1, 2, 1, 4, 24, 1.0, 10000.0), dense(64))], cap=None, eps=1e-6)
# sizes that are multiples of nothing: the bfloat16 products run on zero-padded operands, loads are scalar
CFG_C = config(75, 36, [
    layer(latent(3, 5, 6, 7, 9, 11, 0.4, 100.0, (8.0, 32, 4.0, 1.0)), moe(13, 4, 2)),
    layer(chunked(3, 1, 5, 7, 0.5, 23, True), dense(22)),
    layer(chunked(5, 5, 9, 3, 0.4, 100), moe(11, 7, 4)),
    layer(chunked(2, 1, 13, 7, 0.3, 0, True), dense(15)),
    layer(latent(5, 3, 0, 6, 7, 13, 0.6), None)], cap=3.0)
# sizes that the tensor-core kernels take (the first layer's experts as grouped products): heads of 128 and of 192
# numbers, wide groups of query heads
CFG_D = config(128, 128, [
    layer(latent(8, 64, 64, 64, 96, 256, 0.09, 250000.0, (16.0, 4096, 32.0, 1.0)), moe(128, 8, 2)),
    layer(chunked(12, 2, 128, 128, 0.09, 300, True), dense(256)),
    layer(chunked(20, 1, 64, 32, 0.12, 256), moe(64, 8, 4)),
    layer(chunked(4, 2, 192, 128, 0.07, 500, True), None),
    layer(latent(2, 128, 64, 128, 64, 264, 0.07, 10000.0), dense(128))], cap=30.0)
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}
TAGS = 4          # features that carry a token's class for the routers (see `decisive`)


def bf(t):
    return t.to(torch.bfloat16).to(P.DT)


def decisive(cfg, w):
    """Routers whose choice no rounding turns: the last TAGS features of the residual stream carry the token's class
    (id mod TAGS) from the embedding, no sublayer writes them (the rows of every last product that would are zero), and a
    router reads next to nothing else: every class has its own order of the experts with gaps between their logits."""
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
    for i, lay in enumerate(cfg["layers"]):
        if lay.get("mlp") is None or lay["mlp"]["kind"] != "moe":
            continue
        E = lay["mlp"]["router"]["experts"]
        r = bf(w[f"l{i}.mlp.router"] * 0.004)
        g = torch.Generator().manual_seed(1000 + i)
        for c in range(TAGS):
            order = torch.randperm(E, generator=g)
            r[order, W - TAGS + c] = bf(torch.linspace(-0.7, 0.7, E, dtype=P.DT))
        out[f"l{i}.mlp.router"] = r
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
    assert not P.MARGINS or min(P.MARGINS) > 0.1, min(P.MARGINS)
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
    # the norm's weight is stored around zero: 3 and 4 have mean square 12.5
    x = P.norm_around_one(one(3.0, 4.0), one(0.0, 1.0), 0.0)
    assert torch.allclose(x, one(3.0, 8.0) / math.sqrt(12.5))
    assert torch.allclose(P.relu_squared(one(-3.0, 0.0, 3.0)), one(0.0, 0.0, 9.0))
    assert torch.allclose(P.soft_cap(one(2.0), 4.0), 4.0 * torch.tanh(one(0.5))) and P.soft_cap(one(9.0), None) == 9.0
    # frequencies without scaling: base^(-2 i / dims)
    f, a = P.frequencies(dict(dims=4, base=100.0))
    assert torch.allclose(f, one(1.0, 0.1)) and a == 1.0
    # fast = slow at pair 1.5: lo 1, hi 2; pairs 0 and 1 keep their frequency, pairs 2 and 3 are divided by the factor
    sc = dict(factor=2.0, original=2 * math.pi * math.e ** 0.75, fast=1.0, slow=1.0)
    f, a = P.frequencies(dict(dims=8, base=math.e ** 2, scaling=sc))
    assert torch.allclose(f, one(1.0, math.e ** -0.5, 0.5 * math.e ** -1.0, 0.5 * math.e ** -1.5))
    assert abs(a - (1.0 + 0.1 * math.log(2.0))) < 1e-12
    # rotation pairs number 2 i with 2 i + 1; base 1: every frequency is 1, the angle at position 1 is 1
    y = P.rotate(one(1.0, 2.0, 3.0, 4.0).view(1, 1, 4), torch.tensor([1]), dict(dims=4, base=1.0))
    c, s = math.cos(1.0), math.sin(1.0)
    assert torch.allclose(y.flatten(), one(1 * c - 2 * s, 2 * c + 1 * s, 3 * c - 4 * s, 4 * c + 3 * s))
    # slopes: 2^(-8 (h + 1) / heads)
    assert torch.allclose(P.slopes(4), one(0.25, 0.0625, 2.0 ** -6, 2.0 ** -8)) and float(P.slopes(1)[0]) == 2.0 ** -8
    # the score of position 2 with key 0 (two back): 3 * 0.5 - slope * 2
    q, k = one(0.0, 0.0, 3.0).view(3, 1, 1), one(1.0, 1.0, 1.0).view(3, 1, 1)
    assert abs(float(P.biased_scores(q, k, 0, 0.5)[0, 2, 0]) - (1.5 - 2.0 ** -7)) < 1e-12
    # chunks are counted from position 0, wherever a portion starts
    assert P.visible(5, 2, 7, 3).tolist() == [[False, False, False, True, True, True, False],
                                              [False, False, False, False, False, False, True]]
    assert P.visible(1, 1, 3, None).tolist() == [[True, True, False]]
    # a sink of ln 2 and two keys of score 0: 1/4 each; an unseen key changes nothing
    a = P.softmax_with_sink(one([0.0, 0.0, 5.0]).view(1, 1, 3), torch.tensor([[True, True, False]]), one(math.log(2.0)))
    assert torch.allclose(a.flatten(), one(0.25, 0.25, 0.0))
    assert torch.allclose(P.mix_values(one(2.0), one(10.0), one(0.25)), one(4.0))
    # one gate per head
    o = P.gate_heads({"m.g": one([0.0], [math.log(3.0)])}, "m.", one([1.0]).view(1, 1), torch.ones(1, 2, 3, dtype=P.DT))
    assert torch.allclose(o[0], one([0.5] * 3, [0.75] * 3))
    # the weights are shares of the chosen experts' softmax scores
    chosen, weight = P.choose_experts(one([0.0, math.log(3.0), -5.0, math.log(2.0)]).view(1, 4), 2)
    assert chosen[0].tolist() == [1, 3] and torch.allclose(weight[0], one(0.6, 0.4))


def test_configuration_is_read_by_key_and_written_back():
    from janus_b200.config import ConfigError, resolve_architecture
    for cfg in CONFIGS.values():
        arch = resolve_architecture(cfg)
        c = arch.config_class.from_dict(cfg)
        assert json.loads(json.dumps(c.to_dict())) == json.loads(json.dumps(cfg))
    arch = resolve_architecture(CFG_A)
    c = arch.config_class.from_dict(CFG_A)
    assert [getattr(x.mixer, "chunk", None) for x in c.layers] == [50, None, 37, 128, None, 64]
    assert [getattr(x.mixer, "v_mix", None) for x in c.layers] == [True, None, False, True, None, True]
    assert c.first_mixed == 0 and c.logit_softcap == 8.0 and c.layers[2].mlp is None
    assert c.layers[1].mixer.rot.scaling == (4.0, 64.0, 8.0, 1.0) and c.layers[4].mixer.rot.scaling is None
    b = arch.config_class.from_dict(CFG_B)
    assert b.logit_softcap is None and b.first_mixed == 1
    bare = copy.deepcopy(CFG_A)
    del bare["logit_softcap"], bare["layers"][0]["mixer"]["mask"], bare["layers"][2]["mixer"]["v_mix"]
    c = arch.config_class.from_dict(bare)
    assert c.logit_softcap is None and c.layers[0].mixer.chunk == 0 and not c.layers[2].mixer.v_mix
    for path, value, word in ((("layers", 0, "type"), "gla", "type"), (("layers", 0, "mlp", "kind"), "sparse", "kind"),
                              (("norm",), None, "norm"), (("layers",), [], "layers"),
                              (("layers", 1, "mixer", "rot", "dims"), 4, "dims"), (("layers", 1, "mixer", "rot"), None, "rot"),
                              (("layers", 1, "mixer", "q_rank"), None, "q_rank"), (("layers", 1, "mixer", "kv_rank"), 0, "kv_rank"),
                              (("layers", 1, "mlp", "router", "top"), 7, "top"), (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
                              (("layers", 0, "mixer", "mask", "size"), -4, "size"), (("layers", 3, "mixer", "vdim"), 16, "v_mix"),
                              (("layers", 3, "mixer", "v_mix"), 1, "v_mix"), (("logit_softcap",), 0.0, "logit_softcap"),
                              (("layers", 0, "mixer", "scale"), 0.0, "scale")):
        bad = copy.deepcopy(CFG_A)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            arch.config_class.from_dict(bad)


def test_the_model_description_names_every_tensor_once():
    from janus_b200.config import resolve_architecture
    from janus_b200.engine.model import DecoderModel
    from janus_b200.models.mibezen import distance_slopes, mibezen_spec
    for cfg in CONFIGS.values():
        arch = resolve_architecture(cfg)
        c = arch.config_class.from_dict(cfg)
        names = {s.name: tuple(s.shape) for s in arch.weight_specs(c)}
        want = {k: tuple(v.shape) for k, v in P.random_weights(cfg, 0).items()}
        spec = mibezen_spec(c)
        unread = set(want) - set(names)          # the first mixed layer's share: in the file, read by nothing
        assert unread == {f"l{c.first_mixed}.mix.vmix"} and unread <= set(spec.ignorable_weights)
        assert names == {k: v for k, v in want.items() if k not in unread}
    spec = mibezen_spec(resolve_architecture(CFG_A).config_class.from_dict(CFG_A))
    assert "l2.norm2" in spec.ignorable_weights and spec.layers[2].feed_forward is None
    kv = DecoderModel(spec, torch.bfloat16, torch.device("cpu")).place_cache_specs()
    assert [(s.head_dim, s.v_dim, s.chunk) for s in kv] == [(16, 8, 50), (48, 48, 0), (24, 8, 37), (8, 8, 128), (32, 32, 0),
                                                            (16, 8, 64)]
    spec = mibezen_spec(resolve_architecture(CFG_C).config_class.from_dict(CFG_C))
    bits = [DecoderModel(spec, d, torch.device("cpu")).place_cache_specs()[1] for d in (torch.float32, torch.bfloat16)]
    assert [(s.head_dim, s.v_dim) for s in bits] == [(5, 7), (8, 8)]       # the tensor-core kernels take values up to the keys' size
    assert distance_slopes(4) == tuple(P.slopes(4).tolist()) and distance_slopes(3) == tuple(P.slopes(3).tolist())


def test_rows_are_put_in_the_order_of_the_halves():
    """A rotation of neighbouring pairs is a rotation of halves once the even numbers stand before the odd ones."""
    from janus_b200.parts.latent_attention import RotaryLatentAttention
    m = RotaryLatentAttention(64, 2, 3, 6, 8, 16, 1.0, 1e-5, q_rank=5, pairs="neighbours", gate="head", device=torch.device("cpu"))
    w = torch.arange(18.0).view(18, 1).expand(18, 5)
    assert m._halves(w, 2, 3)[:, 0].tolist() == [0, 1, 2, 3, 5, 7, 4, 6, 8, 9, 10, 11, 12, 14, 16, 13, 15, 17]
    assert m.weight_shapes()["g"][0] == (2, 64) and m.weight_shapes()["uq"][0] == (18, 5)
    plain = RotaryLatentAttention(64, 2, 3, 6, 8, 16, 1.0, 1e-5, device=torch.device("cpu"))
    assert plain._halves(w, 2, 3) is w
    for bad in (dict(gate="row"), dict(pairs="thirds"), dict(q_rank=5, pairs="both")):
        with pytest.raises(ValueError):
            RotaryLatentAttention(64, 2, 3, 6, 8, 16, 1.0, 1e-5, device=torch.device("cpu"), **bad)


def test_pages_of_a_chunk_that_is_over_go_back_to_the_cache():
    from janus_b200.cache import PAGE_SIZE, SequenceCache
    from janus_b200.parts.base import KVSpec
    cache = SequenceCache([KVSpec(1, 8, chunk=100), KVSpec(1, 8)], 64 * 8, 2, torch.float32, torch.device("cpu"))
    held = lambda s: [[p >= 0 for p in g.pages[s]] for g in cache.groups]      # noqa: E731
    slot = cache.alloc_slot()
    for n, want in ((99, [True, True]), (1, [False, True]), (90, [False, True, True]), (20, [False, False, False, True])):
        cache.reserve(slot, n)
        cache.advance(slot, n)
        assert held(slot)[0] == want and all(held(slot)[1]), cache.lengths[slot]
        cache.check()
    other = cache.alloc_slot()
    cache.reserve(other, 3 * PAGE_SIZE)
    cache.advance(other, 3 * PAGE_SIZE)
    cache.check()
    cache.free_slot(slot)
    cache.free_slot(other)
    cache.check()
    assert all(g.pool.n_held == 0 for g in cache.groups)


def far_key_case(seed=6):
    """One layer of latent attention alone and two prompts that differ in their first token only.  Those two tokens (and
    no others) have a feature that makes one latent number large; the last token's query asks for it in every head, so
    what the last position says, 400 tokens on, is the first token's value; the two tokens' other features are
    opposite."""
    cfg = config(64, 32, [layer(latent(2, 8, 4, 8, 12, 16, 0.5, 100.0))])
    w = P.random_weights(cfg, seed)
    m, first_a, first_b, last = "l0.mix.", 0, 1, 2
    emb = w["embed"].clone()
    emb[:, 30:] = 0.0
    emb[first_b, :30] = -emb[first_a, :30]
    emb[first_a, 30] = emb[first_b, 30] = emb[last, 31] = 6.0
    w["embed"] = emb
    for name, row, feature in (("dkv", 0, 30), ("dq", 0, 31)):
        t = w[m + name].clone()
        t[:, 30:] = 0.0
        t[row, :30] = 0.0
        t[row, feature] = 6.0
        w[m + name] = t
    t = w[m + "uq"].clone()
    t[:, 0] = 0.0
    t[[0, 12], 0] = 4.0                        # the first unrotated number of both heads (of 8 + 4 each)
    w[m + "uq"] = bf(t)
    t = w[m + "uk"].clone()
    t[[0, 8], 0] = 3.0
    w[m + "uk"] = t
    t = w[m + "uv"].clone()
    t[:, 0] = 0.0                               # the loud number says nothing itself
    w[m + "uv"] = bf(t * 3.0)
    middle = [3 + t % 61 for t in random_tokens(398, 64, seed)]
    return cfg, w, [first_a] + middle + [last], [first_b] + middle + [last]


def chunk_edge_case(chunk, length, at, seed=8):
    """One attention layer alone and two prompts that differ in the token at position `at` only; both of those tokens are
    loud to the last token's query and their values are opposite."""
    cfg = config(64, 32, [layer(chunked(4, 2, 8, 8, 0.5, chunk))])
    w = P.random_weights(cfg, seed)
    m, loud_a, loud_b, last = "l0.mix.", 0, 1, 2
    emb = w["embed"].clone()
    emb[:, 30:] = 0.0
    emb[loud_b, :30] = -emb[loud_a, :30]
    emb[loud_a, 30] = emb[loud_b, 30] = emb[last, 31] = 6.0
    w["embed"] = emb
    for name, feature, rows in (("k", 30, (0, 8)), ("q", 31, (0, 8, 16, 24))):
        t = w[m + name].clone()
        t[:, 30:] = 0.0
        t[list(rows)] = 0.0
        t[list(rows), feature] = 4.0
        w[m + name] = t
    t = w[m + "v"].clone()
    t[:, 30:] = 0.0
    w[m + "v"] = bf(t * 3.0)
    ids = [3 + t % 61 for t in random_tokens(length, 64, seed)]
    ids[-1] = last
    a, b = list(ids), list(ids)
    a[at], b[at] = loud_a, loud_b
    return cfg, w, a, b


# (chunk, length, place of the loud token, whether the last position sees it)
EDGES = [(50, 100, 50, True), (50, 100, 49, False), (50, 101, 99, False), (64, 128, 64, True), (64, 128, 63, False),
         (100, 191, 100, True), (100, 191, 99, False), (100, 193, 127, True), (100, 193, 128, True), (7, 70, 63, True),
         (7, 70, 62, False), (130, 391, 390 - 130, False), (0, 200, 0, True)]


def test_the_cases_made_to_show_do_show_in_the_plain_logits():
    cfg, w, a, b = far_key_case()
    assert rel_err(plain_logits(cfg, w, a)[-1:], plain_logits(cfg, w, b)[-1:]) > 8 * BF16_TOL
    for chunk, length, at, seen in EDGES:
        cfg, w, a, b = chunk_edge_case(chunk, length, at)
        if at == length - 1:
            continue
        apart = rel_err(plain_logits(cfg, w, a)[-1:], plain_logits(cfg, w, b)[-1:])
        assert apart > 8 * BF16_TOL if seen else apart < 1e-9, (chunk, length, at, apart)
    # what goes wrong without a mechanism moves the logits by more than the bounds
    w = weights_for(CFG_A, 12)
    ids = random_tokens(80, CFG_A["vocab"], 5)
    ref = plain_logits(CFG_A, w, ids)
    keep = {k: getattr(P, k) for k in ("softmax_with_sink", "slopes", "mix_values", "gate_heads", "choose_experts", "rotate",
                                       "visible", "norm_around_one", "relu_squared")}

    def changed(**kw):
        try:
            for k, v in kw.items():
                setattr(P, k, v)
            return P.forward(CFG_A, w, ids)[0]
        finally:
            for k, v in keep.items():
                setattr(P, k, v)

    for kw in (dict(softmax_with_sink=lambda s, seen, sink: keep["softmax_with_sink"](s, seen, torch.full_like(sink, -99.0))),
               dict(softmax_with_sink=lambda s, seen, sink: keep["softmax_with_sink"](s, seen, 0.0 * sink)),
               dict(slopes=lambda H: 0.0 * keep["slopes"](H)), dict(mix_values=lambda v, first, share: v),
               dict(mix_values=lambda v, first, share: share * v + (1.0 - share) * first),
               dict(gate_heads=lambda w_, pre, h, o: o),
               dict(choose_experts=lambda z, top: (z.topk(top).indices, torch.softmax(z, -1).topk(top).values)),
               dict(rotate=lambda x, pos, rot: keep["rotate"](x, pos + (x.shape[1] == 1), rot)),
               dict(visible=lambda start, T, L, chunk: keep["visible"](start, T, L, chunk and chunk + 1)),
               dict(relu_squared=lambda z: torch.clamp(z, min=0.0))):
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
    """Every prompt step of the bfloat16 engine goes this way through latent attention (where its sizes allow)."""
    from janus_b200.parts.latent_attention import RotaryLatentAttention
    monkeypatch.setattr(RotaryLatentAttention, "prompt_way", request.param)
    return request.param


DTYPES_AND_WAYS = [("float32", "latents"), ("bfloat16", "heads"), ("bfloat16", "latents")]
both = pytest.mark.parametrize("dtype,way", DTYPES_AND_WAYS, indirect=["way"])


@gpu
def test_norms_with_weights_stored_around_zero():
    from janus_b200.parts.norm import RMSNorm
    g = torch.Generator().manual_seed(0)
    for T, W in ((7, 64), (5, 37), (300, 2048)):
        x, w = torch.randn(T, W, generator=g) * 3, bf(torch.randn(W, generator=g) * 0.3)
        for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 1e-2)):
            n = RMSNorm(W, 1e-5, weight_offset=1.0, dtype=dtype, device=torch.device("cuda"))
            n.load(w.to(torch.bfloat16))
            out = torch.empty(T, W, dtype=dtype, device="cuda")
            n.forward(x.cuda(), out)
            assert rel_err(out.float().cpu(), P.norm_around_one(x.to(P.DT), w, 1e-5)) < tol


@gpu
def test_products_with_the_squared_relu_in_their_epilogue_and_behind_them():
    from types import SimpleNamespace
    from janus_b200.engine.workspace import Workspace
    from janus_b200.kernels import ops
    from janus_b200.parts.feedforward import SquaredReluFeedForward
    g = torch.Generator().manual_seed(2)
    x = torch.linspace(-6.0, 6.0, 4099)
    out = torch.empty(4099, device="cuda")
    ops.activate(x.cuda(), out, "relu2")
    assert float((out.cpu().to(P.DT) - P.relu_squared(x.to(P.DT))).abs().max()) < 1e-5
    for dtype in (torch.float32, torch.bfloat16):
        for T, W, F in ((3, 64, 200), (70, 96, 136), (300, 256, 512), (20, 36, 50), (9, 256, 20000)):
            h, up, down = (bf(torch.randn(*s, generator=g) * k) for s, k in
                           (((T, W), 1.0), ((F, W), 2.0 * W ** -0.5), ((W, F), F ** -0.5)))
            part = SquaredReluFeedForward(W, F, dtype=dtype)
            part.load(up.to(torch.bfloat16), down.to(torch.bfloat16))
            res = torch.zeros(T, W, device="cuda")
            part.forward(h.to(dtype).cuda(), res, SimpleNamespace(workspace=Workspace(torch.device("cuda"))))
            want = P.dense_ff({"up": up, "down": down}, "", h)
            assert rel_err(res.cpu(), want) < (1e-5 if dtype == torch.float32 else 1.5e-2), (dtype, T, W, F)


@gpu
@pytest.mark.parametrize("H,G,d,e", [(4, 2, 16, 8), (3, 1, 5, 7), (8, 8, 128, 128), (1, 1, 8, 8), (5, 5, 9, 3)])
@pytest.mark.parametrize("extra", [3, 4])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_queries_and_cache_rows_with_values_of_their_own_size_and_a_share_of_others(H, G, d, e, dtype, extra):
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    T, PAGE = 9, 64
    up8 = lambda n: (n + 7) // 8 * 8      # noqa: E731
    ep = up8(e) if dtype == torch.bfloat16 else e
    dp = max(up8(d), ep) if dtype == torch.bfloat16 else d
    tol = 1e-6 if dtype == torch.float32 else 6e-3
    # rows wider than what is read by a whole group of four numbers or not: the kernel for groups of four, and the other one
    proj, other = torch.randn(T, H * d + G * (d + e) + extra, generator=g), torch.randn(T, G * e + 8, generator=g)
    off = extra if extra % 4 == 0 else 2
    dest = torch.tensor([3 * PAGE + 63, 0, 1, 2, PAGE + 7, 5, 2 * PAGE, 63, 64], dtype=torch.int32)
    v = proj[:, (H + G) * d:(H + G) * d + G * e].to(P.DT).view(T, G, e)
    for first, mix in ((None, 0.0), (other.cuda()[:, off:off + G * e], 0.3)):
        kc = torch.zeros(4, G, PAGE, dp, dtype=dtype, device="cuda")
        vc = torch.zeros(4, G, PAGE, ep, dtype=dtype, device="cuda")
        q = torch.full((T, H * dp), 7.0, dtype=dtype, device="cuda")
        ops.head_norm_rope_cache(proj.cuda(), None, None, 1e-5, None, 0, torch.arange(T, dtype=torch.int32).cuda(), q, dest.cuda(),
                                 kc, vc, H, G, d, e, dp, PAGE, stored_vdim=ep, first=first, mix=mix)
        got = q.view(T, H, dp).float().cpu()
        assert rel_err(got[..., :d], proj[:, :H * d].view(T, H, d)) < tol and float(got[..., d:].abs().sum()) == 0.0
        rows = lambda c: c.transpose(1, 2).reshape(4 * PAGE, G, -1).float().cpu()      # noqa: E731
        assert rel_err(rows(kc)[dest.long()][..., :d], proj[:, H * d:(H + G) * d].view(T, G, d)) < tol
        want = v if first is None else P.mix_values(v, other[:, off:off + G * e].to(P.DT).view(T, G, e), torch.tensor(0.3, dtype=P.DT))
        assert rel_err(rows(vc)[dest.long()][..., :e], want) < tol
        idle = [i for i in range(4 * PAGE) if i not in dest.tolist()]
        assert float(rows(vc)[idle].abs().sum()) == 0.0 and float(rows(kc)[idle].abs().sum()) == 0.0


def _case(H, G, hd, vd, lens, q_lens, chunk, g):
    """Sequences whose queries have one loud key each, at the edges of pages, blocks and chunks (just inside and just
    outside); pages handed out of order."""
    PAGE = 64
    n_pages = sum((n + PAGE - 1) // PAGE for n in lens) + 3
    order = iter(torch.randperm(n_pages, generator=g).tolist())
    width = max((n + PAGE - 1) // PAGE for n in lens) + 1
    table = torch.full((len(lens), width), -1, dtype=torch.int32)
    kc, vc = torch.zeros(n_pages, G, PAGE, hd, dtype=P.DT), torch.zeros(n_pages, G, PAGE, vd, dtype=P.DT)
    ks, vs, qs = [], [], []
    for s, (n, ql) in enumerate(zip(lens, q_lens)):
        k, v = bf(torch.randn(n, G, hd, generator=g)), bf(torch.randn(n, G, vd, generator=g))
        for i in range((n + PAGE - 1) // PAGE):
            p = table[s, i] = next(order)
            m = min(PAGE, n - i * PAGE)
            kc[p, :, :m] = k[i * PAGE:i * PAGE + m].transpose(0, 1)
            vc[p, :, :m] = v[i * PAGE:i * PAGE + m].transpose(0, 1)
        q = torch.randn(ql, H, hd, generator=g) * 0.3
        for i in range(ql):
            pos = n - ql + i
            lo = pos // chunk * chunk if chunk else 0
            for h in range(H):
                loud = (pos, lo, max(0, lo - 1), max(0, pos - 1), min(pos, 63), min(pos, 64), min(pos, 128))[(i + 2 * h) % 7]
                q[i, h] = q[i, h] + 1.5 * k[loud, h // (H // G)]
        ks.append(k), vs.append(v), qs.append(bf(q))
    return kc, vc, table, ks, vs, qs


def _wanted(q, k, v, scale, chunk, slopes, sinks, gate):
    """The plain attention with the pieces of `plain_mibezen`; slopes, sinks, gate [T, H] or None."""
    T, H, L = q.shape[0], q.shape[1], k.shape[0]
    start = L - T
    s = P.biased_scores(q, k, start, scale)
    if slopes is None:
        back = torch.arange(start, L)[:, None] - torch.arange(L)[None, :]
        s = s + P.slopes(H)[:, None, None] * back[None].to(P.DT)
    a = P.softmax_with_sink(s, P.visible(start, T, L, chunk), sinks if sinks is not None else torch.full((H,), -math.inf, dtype=P.DT))
    o = torch.einsum("htj,jhe->the", a, v.repeat_interleave(H // v.shape[1], dim=1))
    return o if gate is None else o * torch.sigmoid(gate)[:, :, None]


ATTENTION_SIZES = [(4, 2, 16, 8), (6, 2, 128, 128), (6, 2, 88, 40), (3, 1, 64, 64), (16, 1, 192, 128), (2, 2, 256, 248), (5, 5, 8, 8),
                   (20, 1, 72, 40)]


def _options(H, T, which, g):
    """(slopes, sinks, gate columns): all, or one of them."""
    slopes = P.slopes(H).float() if which in ("all", "slopes") else None
    sinks = torch.randn(H, generator=g) * 2 if which in ("all", "sinks") else None
    gate = torch.randn(T, H + 3, generator=g) if which in ("all", "gate") else None
    return slopes, sinks, gate


def _dt(t):
    return None if t is None else t.to(P.DT)


def _cu(t):
    return None if t is None else t.cuda()


@gpu
@pytest.mark.parametrize("chunk", [0, 50, 128])
@pytest.mark.parametrize("H,G,hd,vd", ATTENTION_SIZES)
def test_prompt_attention_kernels_with_slopes_sinks_gates_and_chunks(H, G, hd, vd, chunk, monkeypatch):
    """Prompts and portions on every kernel that serves them (the two tcgen05 ones, mma.sync, float32), all options
    together and each alone."""
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(5)
    for (lens, q_lens), which in ((([1, 64, 333, 129], [1, 64, 333, 129]), "all"), (([70, 333, 65], [3, 130, 2]), "all"),
                                  (([200], [200]), "slopes"), (([200], [150]), "sinks"), (([200], [64]), "gate")):
        kc, vc, table, ks, vs, qs = _case(H, G, hd, vd, lens, q_lens, chunk, g)
        T, scale = sum(q_lens), 6.0 / hd
        slopes, sinks, gate = _options(H, T, which, g)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32).cuda()      # noqa: E731
        starts = [0] + list(np.cumsum(q_lens))
        want = torch.cat([_wanted(q, k, v, scale, chunk, slopes, _dt(sinks), None if gate is None else gate[a:b, 1:1 + H].to(P.DT))
                          for q, k, v, a, b in zip(qs, ks, vs, starts, starts[1:])])
        kw = dict(chunk=chunk, slopes=_cu(slopes), sinks=_cu(sinks), gate=None if gate is None else gate.cuda()[:, 1:1 + H], vd=vd)
        q = torch.cat(qs).view(T, -1)
        seq = i32([s for s, n in enumerate(q_lens) for _ in range(n)])
        pos = i32([n - m + i for n, m in zip(lens, q_lens) for i in range(m)])
        out32 = torch.empty(T, H * vd, device="cuda")
        ops.attention_f32(q.float().cuda(), kc.float().cuda(), vc.float().cuda(), out32, table.cuda(), seq, pos, H, G, hd, 64, 0, scale,
                          **kw)
        assert rel_err(out32.cpu().view(T, H, vd), want) < 1e-5, (which, lens)
        cache = (kc.to(torch.bfloat16).cuda(), vc.to(torch.bfloat16).cuda())
        args = (table.cuda(), i32(starts), i32(lens), len(lens), max(q_lens), H, G, hd, 64, 0, scale)
        for kind in ("1", "2", "mma"):
            out = torch.full((T, H * vd), 9.0, dtype=torch.bfloat16, device="cuda")
            if kind == "mma":
                ops.attention_bf16_prefill(q.to(torch.bfloat16).cuda(), *cache, out, *args, **kw)
            else:
                monkeypatch.setenv("JANUS_ATTN_TC_TILES", kind)
                ops.attention_tc_prefill(q.to(torch.bfloat16).cuda(), *cache, out, *args, **kw)
            assert rel_err(out.float().cpu().view(T, H, vd), want) < 1.5e-2, (kind, which, lens)
    ops.check_kernel_status(torch.device("cuda"))


@gpu
@pytest.mark.parametrize("chunk", [0, 50, 128])
@pytest.mark.parametrize("H,G,hd,vd", ATTENTION_SIZES)
def test_single_token_attention_with_slopes_sinks_gates_chunks_and_mixed_values(H, G, hd, vd, chunk):
    """One query a sequence, whole and in key splits (some without keys): from queries and pages that are ready, and from
    the projections' accumulators, where the kernel mixes the value and appends it and the key itself."""
    from janus_b200.engine.workspace import Workspace
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(6)
    lens = [1, 64, 65, 700, 33, 129, 101, 100]
    B, scale, mix = len(lens), 6.0 / hd, 0.35
    for which, splits in (("all", None), ("all", 1), ("all", 2), ("all", 5), ("slopes", 1), ("sinks", 2), ("gate", 3)):
        kc, vc, table, ks, vs, qs = _case(H, G, hd, vd, lens, [1] * B, chunk, g)
        slopes, sinks, gate = _options(H, B, which, g)
        kw = dict(chunk=chunk, slopes=_cu(slopes), sinks=_cu(sinks), gate=None if gate is None else gate.cuda()[:, 1:1 + H], vd=vd)
        gates = [None if gate is None else gate[i:i + 1, 1:1 + H].to(P.DT) for i in range(B)]
        kv_len = torch.tensor(lens, dtype=torch.int32).cuda()
        ws = Workspace(torch.device("cuda"))
        bound = min(704, chunk) if chunk else 704
        out = torch.empty(B, H * vd, dtype=torch.bfloat16, device="cuda")
        want = torch.cat([_wanted(q, k, v, scale, chunk, slopes, _dt(sinks), z) for q, k, v, z in zip(qs, ks, vs, gates)])
        k16, v16 = kc.to(torch.bfloat16).cuda(), vc.to(torch.bfloat16).cuda()
        ops.attention_bf16_decode(torch.cat(qs).view(B, -1).to(torch.bfloat16).cuda(), k16, v16, out, table.cuda(), kv_len, H, G, hd, 64,
                                  0, scale, ws, bound, n_splits=splits, **kw)
        assert rel_err(out.float().cpu().view(B, H, vd), want) < 1.5e-2, (which, splits)
        # the same new token from the accumulators: its row of the pages is stale before
        first = torch.randn(B, G * vd + 2, generator=g)
        qkv, dest = torch.zeros(B, H * hd + G * (hd + vd) + 1), []
        mixed = []
        for i, n in enumerate(lens):
            p, r = int(table[i, (n - 1) // 64]), (n - 1) % 64
            dest.append(p * 64 + r)
            qkv[i, :H * hd] = qs[i].reshape(-1).float()
            qkv[i, H * hd:(H + G) * hd] = ks[i][-1].reshape(-1).float()
            qkv[i, (H + G) * hd:-1] = vs[i][-1].reshape(-1).float()
            k16[p, :, r], v16[p, :, r] = 3.0, -3.0
            v = vs[i].clone()
            v[-1] = P.mix_values(v[-1], first[i, 1:1 + G * vd].to(P.DT).view(G, vd), torch.tensor(mix, dtype=P.DT))
            mixed.append(v)
        want = torch.cat([_wanted(q, k, v, scale, chunk, slopes, _dt(sinks), z) for q, k, v, z in zip(qs, ks, mixed, gates)])
        ops.attention_bf16_decode(None, k16, v16, out, table.cuda(), kv_len, H, G, hd, 64, 0, scale, ws, bound, n_splits=splits,
                                  qkv=qkv.cuda(), dest=torch.tensor(dest, dtype=torch.int32).cuda(), first=first.cuda()[:, 1:1 + G * vd],
                                  mix=mix, **kw)
        assert rel_err(out.float().cpu().view(B, H, vd), want) < 1.5e-2, (which, splits)
        for i, n in enumerate(lens):
            p, r = int(table[i, (n - 1) // 64]), (n - 1) % 64
            assert rel_err(k16[p, :, r].float().cpu(), ks[i][-1]) < 1e-6
            assert rel_err(v16[p, :, r].float().cpu(), mixed[i][-1]) < 6e-3


@gpu
@pytest.mark.parametrize("m,r,n", [(20, 8, 40), (9, 6, 11), (1536, 64, 512), (1, 2, 8), (7, 0, 13)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_queries_latent_and_the_row_beside_it(m, r, n, dtype):
    from janus_b200.kernels import ops
    from janus_b200.parts.base import PartSpec, make_part
    g = torch.Generator().manual_seed(4)
    T, PAGE, eps, H = 11, 64, 1e-5, 3
    stored = (n + r + 7) // 8 * 8 if dtype == torch.bfloat16 else n + r
    tol = 3e-6 if dtype == torch.float32 else 1e-2
    positions = torch.tensor([0, 1, 5, 6, 7, 62, 63, 64, 700, 701, 1023])
    sc = dict(factor=4.0, original=100, fast=8.0, slow=1.0)
    table = None
    if r:
        table = make_part("position", PartSpec("ramped_rotary", dict(dims=r, theta=300.0, max_positions=1024, scaling=sc)),
                          torch.float32, torch.device("cuda")).fused_rotary_table()
    proj = torch.randn(T, m + H + n + r, generator=g)
    wa, wc = torch.randn(m, generator=g), torch.randn(n, generator=g)
    # the part as projected holds the even numbers, then the odd ones; the plain rotation wants them interleaved
    p = proj[:, m + H + n:].to(P.DT)
    inter = torch.stack([p[:, :r // 2], p[:, r // 2:]], dim=-1).reshape(T, r)
    turned = P.rotate(inter[:, None], positions, dict(dims=r, base=300.0, scaling=sc) if r else None)[:, 0]
    turned = torch.cat([turned[:, 0::2], turned[:, 1::2]], dim=-1)
    want_row = torch.cat([P.rms_unit(proj[:, m + H:m + H + n].to(P.DT), eps) * wc.to(P.DT), turned], dim=-1)
    dest = torch.tensor([3 * PAGE + 63, 0, 1, 2, PAGE + 7, 5, 2 * PAGE, 63, 64, 70, 100], dtype=torch.int32)
    for with_row in (True, False):
        pages = torch.zeros(4, 1, PAGE, stored, dtype=dtype, device="cuda")
        rows = torch.full((T, stored), 7.0, dtype=dtype, device="cuda")
        a, scratch = torch.empty(T, m, dtype=dtype, device="cuda"), torch.ones(40000, device="cuda")
        row = (m + H, n, stored, wc.cuda(), eps, dest.cuda(), pages) if with_row else None
        ops.latent_down(proj.cuda(), m, wa.cuda(), eps, a, r, table, positions.int().cuda(), row, rows if with_row else None, scratch)
        assert rel_err(a.float().cpu(), P.rms_unit(proj[:, :m].to(P.DT), eps) * wa.to(P.DT)) < tol
        assert float(scratch.abs().sum()) == 0.0
        if with_row:
            flat = pages.view(-1, stored).float().cpu()
            assert rel_err(flat[dest.long(), :n + r], want_row) < tol and rel_err(rows[:, :n + r].float().cpu(), want_row) < tol
            assert float(rows[:, n + r:].abs().sum()) == 0.0 and float(flat[:, n + r:].abs().sum()) == 0.0
        else:
            assert float(pages.abs().sum()) == 0.0


@gpu
def test_gates_per_head_on_values_from_latents_and_on_attention_over_a_matrix(monkeypatch):
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(9)
    for H, n, e in ((4, 40, 24), (3, 11, 7), (2, 512, 128), (5, 8, 1)):
        T, ep = 9, (e + 7) // 8 * 8
        o, uv = bf(torch.randn(T, H, n, generator=g)), bf(torch.randn(H * e, n, generator=g) * n ** -0.5)
        gate = torch.randn(T, H + 2, generator=g)
        want = torch.einsum("thn,hen->the", o, uv.view(H, e, n)) * torch.sigmoid(gate[:, 1:1 + H].to(P.DT))[:, :, None]
        for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 1e-2)):
            out = torch.full((T, H * ep), 9.0, dtype=dtype, device="cuda")
            ops.latent_values(o.to(dtype).cuda().view(T, -1), None, uv.to(dtype).cuda(), gate.cuda()[:, 1:1 + H], out, H, n, e, ep)
            got = out.view(T, H, ep).float().cpu()
            assert rel_err(got[..., :e], want) < tol and float(got[..., e:].abs().sum()) == 0.0
    for tiles in ("1", "2"):
        monkeypatch.setenv("JANUS_ATTN_TC_TILES", tiles)
        for H, hd, vd in ((3, 96, 64), (2, 192, 128)):
            lens, q_lens = [70, 333, 65], [3, 130, 65]
            L, T = sum(lens), sum(q_lens)
            kv, q = bf(torch.randn(L, H * (hd + vd), generator=g)), bf(torch.randn(T, H, hd, generator=g))
            gate = torch.randn(T, H + 1, generator=g)
            k, v = kv[:, :H * hd].view(L, H, hd), kv[:, H * hd:].view(L, H, vd)
            out = torch.empty(T, H * vd, dtype=torch.bfloat16, device="cuda")
            i32 = lambda x: torch.tensor(x, dtype=torch.int32).cuda()      # noqa: E731
            ls, qs = [0] + list(np.cumsum(lens)), [0] + list(np.cumsum(q_lens))
            ops.attention_tc_matrix(q.to(torch.bfloat16).cuda().view(T, -1), kv.to(torch.bfloat16).cuda(), out, i32(ls), i32(qs), i32(lens),
                                    3, 130, H, hd, vd, 333, 6.0 / hd, gate=gate.cuda()[:, 1:])
            want = torch.cat([_wanted(q[a:b], k[c:d], v[c:d], 6.0 / hd, 0, None, None, gate[a:b, 1:].to(P.DT))
                              for a, b, c, d in zip(qs, qs[1:], ls, ls[1:])])
            assert rel_err(out.float().cpu().view(T, H, vd), want) < 1.5e-2
    ops.check_kernel_status(torch.device("cuda"))


@gpu
def test_router_with_weights_that_are_shares_of_their_sum():
    from janus_b200.kernels import ops
    g = torch.Generator().manual_seed(6)
    for T, E, top, scale in ((9, 6, 2, 1.0), (70, 64, 6, 0.5), (1, 1, 1, 1.0), (5, 40, 16, 2.5), (33, 5, 5, 1.0)):
        z = torch.randn(T, E, generator=g) * 3
        wide = torch.cat([z, torch.full((T, 1), 99.0)], dim=1)
        se, sw = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
        ops.route_topk(wide.cuda(), top, se, sw, softmax=True, experts=E, scale=scale, shares=True)
        chosen, weight = P.choose_experts(z.to(P.DT), top)
        assert torch.equal(se.cpu().long(), chosen), (T, E)
        assert rel_err(sw.cpu(), weight * scale) < 1e-5
    # sigmoid scores as shares
    z = torch.tensor([[1.0, -1.0, 0.5]])
    se, sw = torch.empty(1, 2, dtype=torch.int32, device="cuda"), torch.empty(1, 2, device="cuda")
    ops.route_topk(z.cuda(), 2, se, sw, shares=True)
    s = torch.sigmoid(z[0, [0, 2]].to(P.DT))
    assert se.tolist() == [[0, 2]] and rel_err(sw.cpu()[0], s / s.sum()) < 1e-6


# ------------------------------------------------------------------------------------------------
# on the device: the engine
# ------------------------------------------------------------------------------------------------
@gpu
@both
@pytest.mark.parametrize("name,which", [("A", 0), ("A", 1), ("A", 2), ("B", 1), ("C", 0), ("C", 1), ("C", 4), ("D", 0), ("D", 1), ("D", 2),
                                        ("D", 3)])
def test_each_mixer_alone_in_a_layer_without_feed_forward(tmp_path, name, which, dtype, way):
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
    for turn, lengths in enumerate(((140, 75, 20), (90, 130, 129))):
        seqs = [random_tokens(n, cfg["vocab"], 7 * turn + n) for n in lengths]
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
            assert rel_err(torch.cat(got[i]), ref[i]) < tol_for(dtype), (turn, i)
        model.engine.cache.check()
    model.check()


def drawn_config(seed):
    """A configuration drawn from a seed: two to six layers of both kinds, feed-forward or none, sizes that are multiples
    of nothing as often as not."""
    r = np.random.RandomState(seed)
    pick = lambda *xs: xs[r.randint(len(xs))]  # noqa: E731
    layers = []
    mixed_heads, mixed_vdim = int(pick(1, 2, 3)), int(pick(5, 8, 24))
    for i in range(r.randint(2, 7)):
        d, e = int(pick(4, 8, 10, 16, 24, 40)), int(pick(4, 8, 9, 16, 24, 32))
        scale = float(pick(0.3, 0.5, 0.8)) * 8 ** -0.5
        if r.randint(2):
            n, rot = [(40, 8), (11, 6), (24, 2), (8, 8)][r.randint(4)]
            mx = latent(int(pick(1, 2, 3, 4, 5, 8)), d, rot, e, int(pick(6, 16, 21, 40)), n, scale, float(pick(50.0, 10000.0)),
                        pick(None, _YARN, (2.0, 300, 16.0, 2.0)))
        else:
            mix = bool(r.randint(2))
            G = mixed_heads if mix else int(pick(1, 2, 3))
            mx = chunked(G * int(pick(1, 2, 4)), G, d, mixed_vdim if mix else e, scale, int(pick(3, 16, 33, 64, 100, 1000)), mix)
        kind = r.randint(4)
        if kind == 0:
            mlp = None
        elif kind == 1:
            mlp = dense(int(pick(24, 40, 64, 100)))
        else:
            E = int(pick(1, 2, 3, 5, 8))
            mlp = moe(int(pick(16, 24, 33, 64)), E, 1 + r.randint(min(E, 4)))
        layers.append(layer(mx, mlp))
    return config(int(pick(50, 97, 128)), int(pick(32, 40, 64, 72, 36, 128)), layers, cap=pick(None, 5.0, 30.0),
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
@pytest.mark.parametrize("chunk,length,at,seen", EDGES)
def test_keys_just_inside_and_just_outside_a_chunk(tmp_path, chunk, length, at, seen, dtype):
    """A loud key at the edge of a chunk: in one prompt, with the last token decoded, with a portion that begins at the
    edge or inside the chunk, with many decoded tokens."""
    from janus_b200.engine import StepEntry
    cfg, w, a, b = chunk_edge_case(chunk, length, at)
    d = P.save_folder(cfg, w, str(tmp_path / "edge"))
    model = load(d, dtype, max_tokens=1024, max_slots=2)
    for ids in (a, b):
        ref = plain_logits(cfg, w, ids)[-1:]
        for cuts in ([length], [length - 1, 1], [at or 1, length - (at or 1)], [at + 1, length - at - 1], [length - 3, 2, 1],
                     [max(1, length - 45)] + [1] * (length - max(1, length - 45))):
            slot, done = model.alloc_slot(), 0
            for n in [n for n in cuts if n]:
                last = done + n == length
                out = model.step([StepEntry(slot, ids[done:done + n], [n - 1] if last else [])])
                done += n
            assert done == length and rel_err(out.cpu(), ref) < (5 * FP32_TOL if dtype == "float32" else tol_for(dtype)), cuts
            model.free_slot(slot)
    model.check()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_loud_sink_takes_most_of_the_first_tokens_attention(tmp_path, dtype):
    """Sinks of several sizes, among them one far above every score and one far below: the first tokens of a sequence, of
    a chunk and of a portion."""
    from janus_b200.engine import StepEntry
    cfg = config(64, 40, [layer(chunked(4, 1, 8, 16, 0.35, 30), None)])
    w = P.random_weights(cfg, 4)
    w["l0.mix.sink"] = bf(torch.tensor([30.0, -30.0, 1.5, 4.0], dtype=P.DT))
    d = P.save_folder(cfg, w, str(tmp_path / "sink"))
    model = load(d, dtype, max_tokens=512, max_slots=2)
    ids = random_tokens(70, 64, 3)
    ref = plain_logits(cfg, w, ids)
    quiet = dict(w)
    quiet["l0.mix.sink"] = w["l0.mix.sink"] * 0.0
    assert rel_err(P.forward(cfg, quiet, ids)[0], ref) > 3 * BF16_TOL
    for cuts in ([70], [1, 1, 1, 27, 1, 1, 38], [2, 28, 2, 28, 10]):
        slot, at, rows = model.alloc_slot(), 0, []
        for n in cuts:
            rows.append(model.step([StepEntry(slot, ids[at:at + n], range(n))]).cpu())
            at += n
        assert rel_err(torch.cat(rows), ref) < tol_for(dtype), cuts
        model.free_slot(slot)
    model.check()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_from_the_first_token(tmp_path, name, dtype):
    """200 single tokens from position 0 on (pages fill, new ones are taken, those of finished chunks go back), two
    sequences a step, one of them a few tokens behind."""
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
    model.engine.cache.check()
    model.check()


@gpu
@both
def test_a_long_prompt_in_one_step_and_in_portions(tmp_path, dtype, way):
    """700 tokens over eleven pages and several chunks; then the same prompt in portions of 300, 257 and 143 tokens on a
    slot that was used before, beside a second request."""
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
    prompts = [random_tokens(n, CFG_A["vocab"], 3 + n) for n in (5, 70, 1, 33, 48)]
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
    assert cfg2["layers"][2]["mlp"]["router"]["experts"] == 4 and set(w2) == set(P.random_weights(CFG_B, 0)) - {"l1.mix.vmix"}
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
