"""The Nezolorn decoder restated plainly: one function per mechanism, whole sequences, no cache, loops over tokens
where the design has a recurrence.  It shares no code with the package; the tests compare the engine with it.

    x0 = E[token] * embedding.scale + B[(previous token * mul_prev + token * mul_cur) mod buckets]
                                                        (a sequence's first token reads the table's last row)
    x += m * mixer(ln(x) w1);  x += m * ff(ln(x) w2)    ln(z) = (z - mean z) / sqrt(var z + eps), m = residual_mult
    logits = head (ln(x) w_final)

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


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def logsigmoid(z):
    return torch.where(z < 0, z, torch.zeros_like(z)) - torch.log1p(torch.exp(-z.abs()))


# ---- embedding ------------------------------------------------------------------------------------------------------
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Which row of the pair table each token of a sequence reads."""
    rows = [buckets]
    for a, b in zip(tokens[:-1], tokens[1:]):
        rows.append((int(a) * mul_prev + int(b) * mul_cur) % buckets)
    return rows[:len(tokens)]


def embed(cfg, W, tokens):
    e = cfg["embedding"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * e["scale"]
    b = e.get("bigram")
    if b is not None:
        x = x + W["bigram"][torch.tensor(bigram_rows(list(tokens), b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


# ---- rotation ---------------------------------------------------------------------------------------------------------
def rotary_frequency(i, dims, base, scaling=None):
    """Angle per position of pair i.  With `scaling` pairs whose wavelength is long against the original context
    turn `factor` times slower, short ones as they are, those between are blended."""
    f = base ** (-2.0 * i / dims)
    if not scaling:
        return f
    wave = 2.0 * math.pi / f
    original, low, high, factor = (float(scaling[k]) for k in ("original", "low", "high", "factor"))
    if wave < original / high:
        return f
    if wave > original / low:
        return f / factor
    s = (original / wave - low) / (high - low)
    return (1.0 - s) * f / factor + s * f


def rotate_halves(x, positions, dims, base, scaling=None):
    """x [T, heads, d]; dimensions i and i + dims/2 turn together."""
    if not dims:
        return x
    f = torch.tensor([rotary_frequency(i, dims, base, scaling) for i in range(dims // 2)], dtype=x.dtype)
    ang = positions.to(x.dtype)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


# ---- attention over a window and the means of the blocks behind it -----------------------------------------------------
def pooled_window_keys(k, v, i, size, pool):
    """(keys [n, G, d], values) that the query at position i sees: the last `size` tokens and the mean of every block
    of `pool` tokens that lies wholly before them."""
    first = max(0, i - size + 1)
    ks, vs = [k[first:i + 1]], [v[first:i + 1]]
    b = 0
    while pool and b * pool + pool - 1 <= i - size:
        ks.append(k[b * pool:(b + 1) * pool].mean(0, keepdim=True))
        vs.append(v[b * pool:(b + 1) * pool].mean(0, keepdim=True))
        b += 1
    return torch.cat(ks), torch.cat(vs)


def pooled_attention_heads(q, k, v, size, pool, scale):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    n_b = T // pool if pool else 0
    K = torch.cat([k] + [k[b * pool:(b + 1) * pool].mean(0, keepdim=True) for b in range(n_b)])
    V = torch.cat([v] + [v[b * pool:(b + 1) * pool].mean(0, keepdim=True) for b in range(n_b)])
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = (j <= i) & (i - j < size)
    if n_b:
        seen = torch.cat([seen, (torch.arange(n_b)[None, :] + 1) * pool - 1 <= i - size], 1)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ K[:, h // rep].T) * scale
        s = torch.where(seen, s, torch.full_like(s, -math.inf))
        out[:, h] = torch.softmax(s, -1) @ V[:, h // rep]
    return out


def pooled_attention(h, W, m, positions):
    """The left side: one projection makes the keys and, before they turn, the values."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W["q"].T).reshape(T, H, d)
    k = (h @ W["k"].T).reshape(T, G, d)
    v = k
    rot = m.get("rot")
    if rot:
        q = rotate_halves(q, positions, rot["dims"], rot["base"], rot.get("scaling"))
        k = rotate_halves(k, positions, rot["dims"], rot["base"], rot.get("scaling"))
    mask = m.get("mask") or {}
    out = pooled_attention_heads(q, k, v, mask.get("size") or T + 1, mask.get("pool") or 0, m["scale"])
    return out.reshape(T, -1) @ W["o"].T


# ---- matrix memory with exponential gates ------------------------------------------------------------------------------
def matrix_memory_scan(q, k, v, i, f):
    """q, k [T, d], v [T, dv], log gates i, f [T] of one head (q already scaled) -> o [T, dv]."""
    T, d = q.shape
    S = torch.zeros(d, v.shape[1], dtype=q.dtype)
    n = torch.zeros(d, dtype=q.dtype)
    m = torch.zeros((), dtype=q.dtype)
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        m = m_new
        S = keep * S + put * k[t][:, None] * v[t][None, :]
        n = keep * n + put * k[t]
        out[t] = (S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return out


def matrix_memory(h, W, m, eps):
    """The right side."""
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W["q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ W["k"].T).reshape(T, H, d)
    v = (h @ W["v"].T).reshape(T, H, dv)
    i = cap * torch.tanh((h @ W["i"].T + W["i.b"]) / cap)
    f = logsigmoid(cap * torch.tanh((h @ W["f"].T + W["f.b"]) / cap))
    o = torch.stack([matrix_memory_scan(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n]) for n in range(H)], 1)
    o = over_rms(o, eps).reshape(T, H * dv) * W["norm"] * torch.sigmoid(h @ W["g"].T)
    return o @ W["o"].T


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def parallel(h, W, m, positions, eps):
    return m["left_scale"] * pooled_attention(h, sub(W, "left."), m["left"], positions) + \
        m["right_scale"] * matrix_memory(h, sub(W, "right."), m["right"], eps)


# ---- the generalized delta rule ------------------------------------------------------------------------------------------
def general_delta_scan(r, k, v, w, a):
    """All [T, d] of one head: S_t = diag(w) S - (a u)(u^T S) + k v^T (the old S in both); o = S_t^T r."""
    T, d = r.shape
    S = torch.zeros(d, v.shape[1], dtype=r.dtype)
    out = torch.zeros(T, v.shape[1], dtype=r.dtype)
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        S = w[t][:, None] * S - (a[t] * u)[:, None] * (u @ S)[None, :] + k[t][:, None] * v[t][None, :]
        out[t] = S.T @ r[t]
    return out


def general_delta(h, W, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    heads = lambda z: z.reshape(T, H, d)
    r, k, v = (heads(h @ W[n].T) for n in ("r", "k", "v"))
    w = heads(torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ W["w1"].T) @ W["w2"].T + W["w0"])))
    a = heads(torch.sigmoid(h @ W["a"].T + W["a.b"]))
    o = torch.stack([general_delta_scan(r[:, n], k[:, n], v[:, n], w[:, n], a[:, n]) for n in range(H)], 1)
    o = over_rms(o, eps).reshape(T, H * d) * W["norm"] * torch.sigmoid(h @ W["g"].T)
    return o @ W["o"].T


# ---- feed-forward --------------------------------------------------------------------------------------------------------
def dense_ff(h, W):
    g = h @ W["gate"].T
    return (g * torch.sigmoid(g) * (h @ W["up"].T)) @ W["down"].T


# ---- the model -------------------------------------------------------------------------------------------------------------
def forward(cfg, weights, tokens, dtype=torch.float64, return_layers=False):
    """Logits [T, vocab] of one whole sequence (positions 0 .. T-1)."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    positions = torch.arange(len(tokens))
    x = embed(cfg, W, tokens)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, W[p + "norm1"], eps)
        mix = sub(W, p + "mix.")
        if layer["type"] == "parallel":
            x = x + mult * parallel(h, mix, layer["mixer"], positions, eps)
        elif layer["type"] == "general_delta":
            x = x + mult * general_delta(h, mix, layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            x = x + mult * dense_ff(layer_norm(x, W[p + "norm2"], eps), sub(W, p + "mlp."))
        after.append(x)
    logits = layer_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, torch.stack(after)) if return_layers else logits
