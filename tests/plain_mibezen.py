"""A plain, slow implementation of the Mibezen decoder on the CPU: one function per mechanism, written from the
design's equations, sharing no code with the library.  Everything runs in one dtype (float64); the mixers take and
return an explicit state (the latents and rotated key parts, or the keys and values so far), so that the tests can run a
sequence in one piece, in portions or token by token and compare.

Notation: T tokens, W width, H query heads, G key/value heads, d query/key size (of latent attention: its unrotated part),
r rotated numbers, e value size, m size of the queries' latent, n size of the keys' and values' latent, E experts.
Linear weights are [out, in] and applied as W x.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import torch

DT = torch.float64


def read_folder(model_dir: str):
    """config.json and the tensors of model.safetensors (an independent reader of the file format)."""
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        raw = f.read()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    data = raw[8 + n:]
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    out: Dict[str, torch.Tensor] = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        a, b = meta["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[meta["dtype"]]).reshape(meta["shape"]).clone()
        out[name] = t.to(DT) if t.is_floating_point() else t
    return cfg, out


# ---------------------------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------------------------
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_one(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The layers' norm: the stored weight is what a feature's factor differs from one by."""
    return rms_unit(x, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


def soft_cap(z: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return z if cap is None else cap * torch.tanh(z / cap)


# ---------------------------------------------------------------------------------------------
# rotation of neighbouring pairs with ramped frequencies
# ---------------------------------------------------------------------------------------------
def frequencies(rot: dict):
    """(frequency of every pair, factor on cos and sin).  Plain: base^(-2 i / dims) and 1.  Scaled: a frequency goes
    over from its own value to 1/factor of it along a ramp in the pair's number, between the pair that makes `fast`
    turns over the original length and the one that makes `slow`; cos and sin grow by 1 + ln(factor) / 10."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return torch.tensor(f, dtype=DT), 1.0

    def pair_of(turns: float) -> float:
        return dims * math.log(sc["original"] / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair_of(sc["fast"])), 0), min(math.ceil(pair_of(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi * (1.0 - ramp) + fi * ramp / sc["factor"])
    return torch.tensor(out, dtype=DT), 1.0 + 0.1 * math.log(sc["factor"])


def rotate(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, r]: numbers 2 i and 2 i + 1 are a pair, (u, v) -> (u c - v s, v c + u s) by the angle
    position * frequency of pair i; numbers from `dims` on pass unchanged."""
    if rot is None:
        return x
    f, amplitude = frequencies(rot)
    angle = positions.to(DT)[:, None] * f[None, :]
    c, s = torch.cos(angle)[:, None, :] * amplitude, torch.sin(angle)[:, None, :] * amplitude
    out = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * c - v * s
    out[..., 1:rot["dims"]:2] = v * c + u * s
    return out


# ---------------------------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------------------------
def latents(p: dict, w, pre: str, h: torch.Tensor, start: int, eps: float):
    """What a layer keeps of every token: the normed latent c [T, n] and the rotated key part [T, r]."""
    T, n = h.shape[0], p["kv_rank"]
    both = h @ w[pre + "dkv"].T
    c = rms_unit(both[:, :n], eps) * w[pre + "dkv.norm"]
    part = rotate(both[:, None, n:], torch.arange(start, start + T), p.get("rot"))[:, 0]
    return c, part


def latent_queries(p: dict, w, pre: str, h: torch.Tensor, start: int, eps: float) -> torch.Tensor:
    """Queries [T, H, d + r] by way of a latent of their own, the last r numbers of a head rotated."""
    T, H, d, r = h.shape[0], p["heads"], p["dim"], p["rot_dim"]
    a = rms_unit(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]
    q = (a @ w[pre + "uq"].T).view(T, H, d + r)
    return torch.cat([q[..., :d], rotate(q[..., d:], torch.arange(start, start + T), p.get("rot"))], dim=-1)


def gate_heads(w, pre: str, h: torch.Tensor, o: torch.Tensor) -> torch.Tensor:
    """o [T, H, e] times one number per head, the sigmoid of a row of a matrix times the mixer's input."""
    return o * torch.sigmoid(h @ w[pre + "g"].T)[:, :, None]


def latent_attention(p: dict, w, pre: str, h: torch.Tensor, start: int, c: torch.Tensor, part: torch.Tensor,
                     eps: float) -> torch.Tensor:
    """h [T, W] at positions start ..; c [start + T, n] and part [start + T, r] of the sequence from position 0 on."""
    T, L, H, d, r, e = h.shape[0], c.shape[0], p["heads"], p["dim"], p["rot_dim"], p["vdim"]
    q = latent_queries(p, w, pre, h, start, eps)
    k = torch.cat([(c @ w[pre + "uk"].T).view(L, H, d), part[:, None, :].expand(L, H, r)], dim=-1)
    v = (c @ w[pre + "uv"].T).view(L, H, e)
    s = torch.einsum("thd,jhd->htj", q, k) * p["scale"]
    seen = torch.arange(L)[None, :] <= torch.arange(start, start + T)[:, None]
    a = torch.softmax(s.masked_fill(~seen[None], -math.inf), dim=-1)
    o = torch.einsum("htj,jhe->the", a, v)
    return gate_heads(w, pre, h, o).reshape(T, H * e) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------
# attention with a distance bias, chunks, a sink and mixed values
# ---------------------------------------------------------------------------------------------
def slopes(H: int) -> torch.Tensor:
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=DT)


def mix_values(v: torch.Tensor, first: torch.Tensor, share: torch.Tensor) -> torch.Tensor:
    return (1.0 - share) * v + share * first


def keys_and_values(p: dict, w, pre: str, h: torch.Tensor):
    T, G = h.shape[0], p["kv_heads"]
    return (h @ w[pre + "k"].T).view(T, G, p["dim"]), (h @ w[pre + "v"].T).view(T, G, p["vdim"])


def visible(start: int, T: int, L: int, chunk: Optional[int]) -> torch.Tensor:
    """[T, L]: position start + t sees j <= it in its own chunk of positions (no chunk: every j <= it)."""
    i, j = torch.arange(start, start + T)[:, None], torch.arange(L)[None, :]
    seen = j <= i
    return seen if not chunk else seen & (i // chunk == j // chunk)


def biased_scores(q, k, start: int, scale: float) -> torch.Tensor:
    """[H, T, L]: the scaled product less the head's slope times how far the key lies back; q [T, H, d], k [L, G, d]."""
    T, H, L = q.shape[0], q.shape[1], k.shape[0]
    k = k.repeat_interleave(H // k.shape[1], dim=1)
    back = torch.arange(start, start + T)[:, None] - torch.arange(L)[None, :]
    return torch.einsum("thd,jhd->htj", q, k) * scale - slopes(H)[:, None, None] * back[None].to(DT)


def softmax_with_sink(s: torch.Tensor, seen: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """s [H, T, L], seen [T, L], sink [H]: weights e^s / (e^sink + sum e^s) of the keys that are seen."""
    s = s.masked_fill(~seen[None], -math.inf)
    extra = sink[:, None, None].expand(s.shape[0], s.shape[1], 1)
    return torch.softmax(torch.cat([s, extra], dim=-1), dim=-1)[..., :-1]


def attention(p: dict, w, pre: str, h: torch.Tensor, start: int, k: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
    """h [T, W] at positions start ..; k [start + T, G, d] and v [start + T, G, e] (mixed) from position 0 on."""
    T, H, e = h.shape[0], p["heads"], p["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, p["dim"])
    chunk = (p.get("mask") or {}).get("size")
    a = softmax_with_sink(biased_scores(q, k, start, p["scale"]), visible(start, T, k.shape[0], chunk), w[pre + "sink"])
    o = torch.einsum("htj,jhe->the", a, v.repeat_interleave(H // p["kv_heads"], dim=1))
    return gate_heads(w, pre, h, o).reshape(T, H * e) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------------------------
def dense_ff(w, pre: str, h: torch.Tensor) -> torch.Tensor:
    return relu_squared(h @ w[pre + "up"].T) @ w[pre + "down"].T


def one_expert(w, pre: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


MARGINS: List[float] = []       # the smallest gap of router logits that a choice of experts rested on, per call


def choose_experts(z: torch.Tensor, top: int):
    """z [T, E] router logits: the `top` largest of the softmax over all experts, as shares of their own sum."""
    ranked, order = torch.softmax(z, dim=-1).sort(dim=-1, descending=True)
    if top < z.shape[1]:
        by_size = z.sort(dim=-1, descending=True).values
        MARGINS.append(float((by_size[:, top - 1] - by_size[:, top]).min()))
    best = ranked[:, :top]
    return order[:, :top], best / (best.sum(dim=-1, keepdim=True) + 1e-20)


def expert_ff(m: dict, w, pre: str, h: torch.Tensor) -> torch.Tensor:
    r = m["router"]
    chosen, weight = choose_experts(h @ w[pre + "router"].T, r["top"])
    out = torch.zeros_like(h)
    for x in range(r["experts"]):
        t, j = (chosen == x).nonzero(as_tuple=True)
        if len(t):
            out[t] += weight[t, j][:, None] * one_expert(w, f"{pre}e{x}.", h[t])
    return out


# ---------------------------------------------------------------------------------------------
# the whole model
# ---------------------------------------------------------------------------------------------
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], state: Optional[dict] = None, start: int = 0,
            layers_out: Optional[list] = None):
    """Logits [T, vocab] of `tokens` at positions start .., from `state` (None: a sequence's beginning), and the
    state after them.  `layers_out` collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    kept, first = {}, None
    for i, layer in enumerate(cfg["layers"]):
        pre, p = f"l{i}.", layer["mixer"]
        h = norm_around_one(x, w[pre + "norm1"], eps)
        if layer["type"] == "latent_attention":
            new = latents(p, w, pre + "mix.", h, start, eps)
        else:
            k, v = keys_and_values(p, w, pre + "mix.", h)
            if p.get("v_mix"):
                if first is None:
                    first = v
                else:
                    v = mix_values(v, first, w[pre + "mix.vmix"])
            new = (k, v)
        kept[i] = new if state is None else tuple(torch.cat([a, b]) for a, b in zip(state[i], new))
        if layer["type"] == "latent_attention":
            x = x + latent_attention(p, w, pre + "mix.", h, start, *kept[i], eps)
        else:
            x = x + attention(p, w, pre + "mix.", h, start, *kept[i])
        m = layer.get("mlp")
        if m is not None:
            h = norm_around_one(x, w[pre + "norm2"], eps)
            x = x + (dense_ff(w, pre + "mlp.", h) if m["kind"] == "dense" else expert_ff(m, w, pre + "mlp.", h))
        if layers_out is not None:
            layers_out.append(x.clone())
    return soft_cap(norm_around_one(x, w["final.norm"], eps) @ w["head"].T, cfg.get("logit_softcap")), kept


def greedy(cfg: dict, w, prompt: List[int], n: int) -> List[int]:
    logits, state = forward(cfg, w, prompt)
    out, pos = [], len(prompt)
    for _ in range(n):
        out.append(int(torch.argmax(logits[-1])))
        logits, state = forward(cfg, w, out[-1:], state, pos)
        pos += 1
    return out


def forward_in_pieces(cfg: dict, w, tokens: List[int], pieces: List[int]) -> torch.Tensor:
    """The same logits, the tokens fed in portions of the given sizes from the state the portions before left."""
    out, state, at = [], None, 0
    for n in pieces:
        logits, state = forward(cfg, w, tokens[at:at + n], state, at)
        out.append(logits)
        at += n
    assert at == len(tokens)
    return torch.cat(out)


# ---------------------------------------------------------------------------------------------
# random weights and model folders
# ---------------------------------------------------------------------------------------------
def random_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Random tensors for a configuration, rounded to bfloat16 values (as a stored model's are)."""
    g = torch.Generator().manual_seed(seed)
    W = int(cfg["width"])

    def rnd(*shape, s=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * s + mean).to(torch.bfloat16).to(DT)

    def mat(rows, cols, s=1.0):
        return rnd(rows, cols, s=s * cols ** -0.5)

    w = {"embed": rnd(cfg["vocab"], W), "head": mat(cfg["vocab"], W, 2.0), "final.norm": rnd(W, s=0.2)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, mx = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        H, d, e = mx["heads"], mx["dim"], mx["vdim"]
        w[p + "norm1"] = rnd(W, s=0.2)
        if layer["type"] == "latent_attention":
            r, a, n = mx["rot_dim"], mx["q_rank"], mx["kv_rank"]
            w[m + "dq"], w[m + "dq.norm"], w[m + "uq"] = mat(a, W), rnd(a, s=0.1, mean=1.0), mat(H * (d + r), a, 1.5)
            w[m + "dkv"], w[m + "dkv.norm"] = mat(n + r, W), rnd(n, s=0.1, mean=1.0)
            w[m + "uk"], w[m + "uv"] = mat(H * d, n), mat(H * e, n)
        else:
            G = mx["kv_heads"]
            w[m + "q"], w[m + "k"], w[m + "v"] = mat(H * d, W, 1.5), mat(G * d, W), mat(G * e, W)
            w[m + "sink"] = rnd(H, s=1.0, mean=0.5)
            if mx.get("v_mix"):
                w[m + "vmix"] = (torch.rand((), generator=g) * 0.6 + 0.2).to(torch.bfloat16).to(DT)
        w[m + "g"], w[m + "o"] = mat(H, W), mat(W, H * e, 1.5)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        w[p + "norm2"] = rnd(W, s=0.2)
        if mlp["kind"] == "dense":
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(mlp["ff"], W), mat(W, mlp["ff"], 0.8)
            continue
        E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        w[p + "mlp.router"] = rnd(E, W, s=2.0 * W ** -0.5)
        for x in range(E):
            q = f"{p}mlp.e{x}."
            w[q + "gate"], w[q + "up"], w[q + "down"] = mat(F, W), mat(F, W), mat(W, F, 1.5)
    return w


def save_folder(cfg: dict, w: Dict[str, torch.Tensor], out_dir: str, dtype=torch.bfloat16) -> str:
    """Write config.json and model.safetensors (an independent writer of the file format)."""
    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    names = {torch.bfloat16: "BF16", torch.float32: "F32"}
    for name, t in w.items():
        t = t.to(dtype).contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": names[dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(os.path.join(out_dir, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return out_dir
