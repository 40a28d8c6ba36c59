"""A plain, slow implementation of the Forisun decoder on the CPU: one function per mechanism, written from the
design's equations, sharing no code with the library.  Everything runs in one dtype (float64); the mixer takes and
returns an explicit state (the latents and rotated key parts so far), so that the tests can run a sequence in one
piece, in portions or token by token and compare.

Notation: T tokens, W width, H heads, d unrotated and r rotated query/key numbers per head, e value size, n latent size,
E experts.  Linear weights are [out, in] and applied as W x.
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
def squash(x: torch.Tensor, alpha: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """The design's norm: no mean and no variance, tanh(alpha x) w + b feature by feature."""
    return torch.tanh(alpha * x) * w + b


def norm(w: Dict[str, torch.Tensor], name: str, x: torch.Tensor) -> torch.Tensor:
    return squash(x, w[name + ".alpha"], w[name], w[name + ".b"])


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu(z: torch.Tensor) -> torch.Tensor:
    """z times the normal distribution's cumulative probability at z."""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ---------------------------------------------------------------------------------------------
# rotation with ramped frequencies
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
    """x [T, heads, r]: number i < dims/2 is paired with i + dims/2, (u, v) -> (u c - v s, v c + u s) by the angle
    position * frequency; numbers from `dims` on pass unchanged."""
    if rot is None:
        return x
    f, amplitude = frequencies(rot)
    half = rot["dims"] // 2
    angle = positions.to(DT)[:, None] * f[None, :]
    c, s = torch.cos(angle)[:, None, :] * amplitude, torch.sin(angle)[:, None, :] * amplitude
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


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


def causal_attention(q, k, v, start: int, scale: float) -> torch.Tensor:
    """q [T, H, .] at positions start ..; k, v [start + T, H, .] from position 0 on.  Position i sees every j <= i."""
    T, H = q.shape[0], q.shape[1]
    s = torch.einsum("thd,jhd->htj", q, k) * scale
    seen = torch.arange(k.shape[0])[None, :] <= torch.arange(start, start + T)[:, None]
    a = torch.softmax(s.masked_fill(~seen[None], -math.inf), dim=-1)
    return torch.einsum("htj,jhe->the", a, v)


def latent_attention(p: dict, w, pre: str, h: torch.Tensor, start: int, c: torch.Tensor, part: torch.Tensor) -> torch.Tensor:
    """h [T, W] at positions start ..; c [start + T, n] and part [start + T, r] of the sequence from position 0 on."""
    T, L, H, d, r, e = h.shape[0], c.shape[0], p["heads"], p["dim"], p["rot_dim"], p["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], torch.arange(start, start + T), p.get("rot"))], dim=-1)
    k = torch.cat([(c @ w[pre + "uk"].T).view(L, H, d), part[:, None, :].expand(L, H, r)], dim=-1)
    v = (c @ w[pre + "uv"].T).view(L, H, e)
    o = causal_attention(q, k, v, start, p["scale"]).reshape(T, H * e)
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------------------------
def dense_ff(w, pre: str, h: torch.Tensor) -> torch.Tensor:
    return gelu(h @ w[pre + "up"].T) @ w[pre + "down"].T


def one_expert(w, pre: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


MARGINS: List[float] = []       # the smallest gap of choice scores that a choice of experts rested on, per call


def choose_experts(z: torch.Tensor, correction: torch.Tensor, top: int, scale: float):
    """z [T, E] router logits: the `top` largest of sigmoid(z) + correction are chosen; a chosen expert's weight is
    sigmoid(z) * scale."""
    s = torch.sigmoid(z)
    ranked, order = (s + correction).sort(dim=-1, descending=True)
    if top < z.shape[1]:
        MARGINS.append(float((ranked[:, top - 1] - ranked[:, top]).min()))
    chosen = order[:, :top]
    return chosen, s.gather(1, chosen) * scale


def expert_ff(m: dict, w, pre: str, h: torch.Tensor) -> torch.Tensor:
    r = m["router"]
    chosen, weight = choose_experts(h @ w[pre + "router"].T, w[pre + "correction"], r["top"], r["scale"])
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
    x = norm(w, "embed.norm", w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"])
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        pre, p = f"l{i}.", layer["mixer"]
        h = norm(w, pre + "norm1", x)
        j = p.get("kv_from")
        if j is None:
            c, part = latents(p, w, pre + "mix.", h, start, eps)
            if state is not None:
                c, part = torch.cat([state[i][0], c]), torch.cat([state[i][1], part])
            kept[i] = (c, part)
        else:
            c, part = kept[j]
        x = x + norm(w, pre + "norm1b", latent_attention(p, w, pre + "mix.", h, start, c, part))
        m = layer.get("mlp")
        if m is not None:
            h = norm(w, pre + "norm2", x)
            y = dense_ff(w, pre + "mlp.", h) if m["kind"] == "dense" else expert_ff(m, w, pre + "mlp.", h)
            x = x + norm(w, pre + "norm2b", y)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(w, "final.norm", x) @ w["head"].T, kept


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

    def mat(rows, cols):
        return rnd(rows, cols, s=cols ** -0.5)

    w = {"embed": rnd(cfg["vocab"], W), "head": mat(cfg["vocab"], W)}

    def put_norm(name, alpha):
        w[name], w[name + ".b"] = rnd(W, s=0.15, mean=1.0), rnd(W, s=0.15)
        w[name + ".alpha"] = (torch.rand((), generator=g) * 0.4 * alpha + 0.8 * alpha).to(torch.bfloat16).to(DT)

    put_norm("embed.norm", 0.8 / cfg["embedding"]["scale"])
    put_norm("final.norm", 0.5)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mx = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        H, d, r, e, n = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
        put_norm(p + "norm1", 0.7)
        put_norm(p + "norm1b", 1.5)
        w[m + "q"] = mat(H * (d + r), W)
        if mx.get("kv_from") is None:
            w[m + "dkv"], w[m + "dkv.norm"] = mat(n + r, W), rnd(n, s=0.1, mean=1.0)
        w[m + "uk"], w[m + "uv"] = mat(H * d, n), mat(H * e, n)
        w[m + "g"], w[m + "o"] = mat(H * e, W), rnd(W, H * e, s=1.5 * (H * e) ** -0.5)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        put_norm(p + "norm2", 0.7)
        put_norm(p + "norm2b", 1.5)
        if mlp["kind"] == "dense":
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(mlp["ff"], W), mat(W, mlp["ff"])
            continue
        E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        w[p + "mlp.router"], w[p + "mlp.correction"] = rnd(E, W, s=2.0 * W ** -0.5), rnd(E, s=0.4)
        for x in range(E):
            q = f"{p}mlp.e{x}."
            w[q + "gate"], w[q + "up"], w[q + "down"] = mat(F, W), mat(F, W), mat(W, F)
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
