"""The Netolorn decoder restated plainly: one function per mechanism, whole sequences, no cache, masks written out as
matrices.  It shares no code with the package; the tests compare the engine with it.

    x = x0 = E[token]
    layers `loop.start` .. `loop.stop` - 1 run `loop.times` times in a row (same weights, a cache of their own each
    time); before every pass, the first too, x <- W_in [x; x0]; the other layers run once, in order
    x += n1b(mixer(n1(x)));  x += n2b(ff(n2(x)))          n(z) = tanh(alpha z) w + b, one alpha per norm
    x += rms(P( gelu_tanh(G x) * S_i[token] )) w_side       S_i: layer i's columns of the per-token table
    logits = head n_final(x)

`weights` maps tensor names to torch tensors; `cfg` is the dict a config.json of the design holds.  Everything runs
in the dtype of `dtype` (float64 for the yardstick, float32 for its own rounding error).
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch


def read_safetensors(path) -> dict:
    """{name: tensor} of a safetensors file: 8 bytes of length, that many of JSON, then the data."""
    raw = Path(path).read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    meta = json.loads(raw[8:8 + n])
    types = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    out = {}
    for name, m in meta.items():
        if name == "__metadata__":
            continue
        a, b = m["data_offsets"]
        out[name] = torch.frombuffer(bytearray(raw[8 + n + a:8 + n + b]), dtype=types[m["dtype"]]).reshape(m["shape"])
    return out


def read_model_dir(model_dir):
    model_dir = Path(model_dir)
    return json.loads((model_dir / "config.json").read_text()), read_safetensors(model_dir / "model.safetensors")


# ---- norms and small functions ------------------------------------------------------------------------------------
def tanh_norm(x, alpha, w, b):
    """Dynamic Tanh: no mean, no variance."""
    return torch.tanh(alpha * x) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- rotation of halves with frequencies scaled by parts -----------------------------------------------------------
def turn_frequencies(dims, base, scaling=None):
    """([dims/2] angle per position of each pair, factor on cos and sin)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def at(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(at(scaling["fast"])), 0)
    hi = min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x, positions, dims, base, scaling=None):
    """x [T, heads, d]; dimension i of the first `dims` is paired with i + dims/2."""
    if not dims:
        return x
    f, mag = turn_frequencies(dims, base, scaling)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = (torch.cos(ang) * mag).to(x.dtype)[:, None, :], (torch.sin(ang) * mag).to(x.dtype)[:, None, :]
    h = dims // 2
    u, v = x[..., :h], x[..., h:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


# ---- what a query sees, and the softmax ------------------------------------------------------------------------------
def window_mask(T, size=None, keep_first=0):
    """[T, T] bool: query i (row) sees key j <= i if i - j < size, or if j is one of the first `keep_first` tokens."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def softmax_sink(s, seen, sink=None):
    """Softmax over the seen keys; a sink is one more score in the denominator."""
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return e / total


# ---- the mixers ----------------------------------------------------------------------------------------------------------
def attention(h, W, m, positions, eps):
    """Mixer 'attention': biased projections, rotation, q and k over their root mean square per head, a window with
    kept first tokens, a learned sink per head, a gate per output element."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W["q"].T + W["q.b"]).reshape(T, H, d)
    k = (h @ W["k"].T + W["k.b"]).reshape(T, G, d)
    v = (h @ W["v"].T + W["v.b"]).reshape(T, G, dv)
    rot = m.get("rot")
    if rot:
        q = rotate_halves(q, positions, rot["dims"], rot["base"], rot.get("scaling"))
        k = rotate_halves(k, positions, rot["dims"], rot["base"], rot.get("scaling"))
    q, k = rms(q, eps), rms(k, eps)
    mask = m.get("mask") or {}
    seen = window_mask(T, mask.get("size"), mask.get("keep_first", 0))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        out[:, n] = softmax_sink((q[:, n] @ k[:, g].T) * m["scale"], seen, W["sink"][n]) @ v[:, g]
    return (out.reshape(T, H * dv) * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def latent_attention(h, W, m, eps):
    """Mixer 'latent_attention': queries and keys/values through normed latents, no positions, a window, a gate per
    head."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = ((rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T).reshape(T, H, d)
    c = rms(h @ W["dkv"].T, eps) * W["dkv.norm"]
    k = (c @ W["uk"].T).reshape(T, H, d)
    v = (c @ W["uv"].T).reshape(T, H, dv)
    seen = window_mask(T, (m.get("mask") or {}).get("size"))
    gate = torch.sigmoid(h @ W["g"].T)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for n in range(H):
        out[:, n] = softmax_sink((q[:, n] @ k[:, n].T) * m["scale"], seen) @ v[:, n] * gate[:, n:n + 1]
    return out.reshape(T, H * dv) @ W["o"].T


# ---- feed-forwards -------------------------------------------------------------------------------------------------------
def dense_ff(h, W):
    g = h @ W["gate"].T
    return (g * torch.sigmoid(g) * (h @ W["up"].T)) @ W["down"].T


def clamped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, W, r):
    """(chosen experts [T, top], weights [T, top]): the largest biased logits, softmax over the chosen."""
    z = h @ W["router"].T + W["router.b"]
    best = z.topk(r["top"], -1)
    return best.indices, torch.softmax(best.values, -1)


def moe_ff(h, W, mlp):
    idx, w = route(h, W, mlp["router"])
    out = torch.zeros(h.shape[0], W["e0.down"].shape[0], dtype=h.dtype)
    for e in range(mlp["router"]["experts"]):
        t, j = torch.nonzero(idx == e, as_tuple=True)
        if t.numel():
            y = clamped_expert(h[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"], mlp["expert"]["limit"])
            out.index_add_(0, t, y * w[t, j][:, None])
    if mlp.get("shared"):
        y = clamped_expert(h, W["shared.gate"], W["shared.up"], W["shared.down"], mlp["shared"]["limit"])
        out = out + torch.sigmoid(h @ W["shared.sg"].T) * y
    return out


# ---- the per-token input of a layer ----------------------------------------------------------------------------------------
def token_side(x, e, gate, proj, norm, eps):
    """What joins x after the layer's feed-forward; e [T, dim] the layer's columns of the tokens' rows."""
    return rms((gelu_tanh(x @ gate.T) * e) @ proj.T, eps) * norm


# ---- the model -----------------------------------------------------------------------------------------------------------
def layer_order(cfg):
    """[(layer, pass or None)] in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop or loop["stop"] <= loop["start"]:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64, return_layers=False):
    """Logits [T, vocab] of one whole sequence (positions 0 .. T-1)."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    norm = lambda name, z: tanh_norm(z, W[name + ".alpha"], W[name], W[name + ".b"])
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(tokens.numel())
    x = x0 = W["embed"][tokens]
    side = cfg.get("token_side")
    loop = cfg.get("loop") or {}
    after = []
    for i, t in layer_order(cfg):
        if t is not None and i == loop["start"]:
            x = torch.cat([x, x0], -1) @ W["loop.in"].T
        layer, p = cfg["layers"][i], f"l{i}."
        h, mix = norm(p + "norm1", x), sub(W, p + "mix.")
        if layer["type"] == "attention":
            y = attention(h, mix, layer["mixer"], positions, eps)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, mix, layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        x = x + norm(p + "norm1b", y)
        mlp = layer.get("mlp")
        if mlp is not None:
            h, ff = norm(p + "norm2", x), sub(W, p + "mlp.")
            y = dense_ff(h, ff) if mlp["kind"] == "dense" else moe_ff(h, ff, mlp)
            x = x + norm(p + "norm2b", y)
        if side:
            e = W["side.embed"][tokens][:, i * side["dim"]:(i + 1) * side["dim"]]
            x = x + token_side(x, e, W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"], eps)
        after.append(x)
    logits = norm("final.norm", x) @ W["head"].T
    return (logits, torch.stack(after)) if return_layers else logits
