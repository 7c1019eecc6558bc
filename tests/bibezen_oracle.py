"""Plain, slow restatement of the Bibezen design in torch on the CPU — one function per mechanism, written from the
design's equations and sharing no code with the package.  It takes the config as the plain dict config.json holds and the
weights under their checkpoint names (as float tensors).

Bibezen: `streams` copies of the residual stream, all equal to the scaled embedding at the start.  Every sublayer reads a
weighted sum u of the copies, and the copies become a small matrix times the old copies plus a per-copy weight times the
sublayer's output on norm(u) — first the mixer, then the feed-forward.  What a mixer reads is the normed row plus a short causal
convolution of the normed rows.  Mixers: Mamba's selective scan ("mamba1"), RWKV-style time mixing ("wkv"), or the
weighted sum of an attention and a time mixing over the same input ("parallel"); the attention has convolved, normed and
rotated queries and keys, tanh-capped scores, a sliding window with mean-pooled blocks behind it, a sink, and mixes the
heads' weights.  Feed-forwards: a clamped gated unit, or routed gated experts with a shared one.  The embedding table is
also the head.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

W = Dict[str, torch.Tensor]


# --------------------------------------------------------------------------------------------------------------- norms
def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def centred_norm(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose weight is stored as its distance from one."""
    return rms(v, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# --------------------------------------------------------------------------------------------------- short convolutions
def causal_conv(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [T, channels], taps [channels, n]: the last column meets the current row, rows before the first are zero."""
    T, n = u.shape[0], taps.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for back in range(n):
            if t - back >= 0:
                out[t] += taps[:, n - 1 - back] * u[t - back]
    return out


def input_conv(h: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    return h + causal_conv(h, taps)


# -------------------------------------------------------------------------------------------------- hyper-connections
def hc_read(x: torch.Tensor, w: W, p: str) -> torch.Tensor:
    """x [T, streams, width] → the sublayer's input before its norm."""
    return torch.einsum("s,tsw->tw", w[p + "in"], x)


def hc_write(x: torch.Tensor, y: torch.Tensor, w: W, p: str, mult: float) -> torch.Tensor:
    """mix is indexed [from, to]."""
    return torch.einsum("sd,tsw->tdw", w[p + "mix"], x) + mult * w[p + "out"][None, :, None] * y[:, None, :]


# -------------------------------------------------------------------------------------------------------------- rotary
def rotate_half(v: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """v [T, heads, n]: entry i < dims/2 of a head turns with entry i + dims/2; the entries from dims on pass."""
    if dims == 0:
        return v
    half = dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(v.dtype)[:, None, :], torch.sin(ang).to(v.dtype)[:, None, :]
    out = v.clone()
    a, b = v[..., :half], v[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


# ----------------------------------------------------------------------------------------------------------- attention
def attention_qkv(h: torch.Tensor, positions: torch.Tensor, m: dict, w: W, p: str, eps: float):
    """Queries, keys and values as they are attended: projection + bias, convolution, head norms (q, k), rotation (q, k)."""
    T, H, G, dk, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    out = []
    for nm, heads, d in (("q", H, dk), ("k", G, dk), ("v", G, dv)):
        u = h @ w[p + nm].T + w[p + nm + ".b"]
        u = causal_conv(u, w[p + nm + ".conv"]).view(T, heads, d)
        if nm != "v":
            u = rms(u, eps) * w[p + nm + ".norm"]
            if m.get("rot"):
                u = rotate_half(u, positions, int(m["rot"]["dims"]), float(m["rot"]["base"]))
        out.append(u)
    return out


def pooled_blocks(rows: torch.Tensor, pool: int) -> torch.Tensor:
    """rows [T, heads, n] → the mean of every whole block of `pool` consecutive rows."""
    nb = rows.shape[0] // pool
    return rows[:nb * pool].view(nb, pool, rows.shape[1], rows.shape[2]).mean(1)


def visible_tokens(n: int, size: int) -> torch.Tensor:
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i - j < size if size > 0 else torch.ones(n, n, dtype=torch.bool))


def visible_blocks(n: int, nb: int, pool: int, size: int) -> torch.Tensor:
    i, b = torch.arange(n)[:, None], torch.arange(nb)[None, :]
    return b * pool + pool - 1 <= i - size


def attention_weights(q, k_tok, k_blk, m: dict, sink: torch.Tensor, use_sink: bool = True, use_cap: bool = True):
    """Softmax weights [H, T, T + blocks] of the tokens and the pooled blocks together; the denominator also holds exp(sink)."""
    T, H, G = q.shape[0], q.shape[1], k_tok.shape[1]
    size, pool = int(m["mask"]["size"]), int(m["mask"]["pool"])
    vis = torch.cat([visible_tokens(T, size), visible_blocks(T, k_blk.shape[0], pool, size)], 1)
    keys = torch.cat([k_tok, k_blk], 0)
    out = torch.zeros(H, T, keys.shape[0], dtype=q.dtype)
    for hd in range(H):
        s = q[:, hd] @ keys[:, hd // (H // G)].T * float(m["scale"])
        if use_cap:
            s = float(m["softcap"]) * torch.tanh(s / float(m["softcap"]))
        s = s.masked_fill(~vis, float("-inf"))
        mx = s.max(-1, keepdim=True).values
        e = torch.exp(s - mx)
        den = e.sum(-1, keepdim=True)
        if use_sink:
            den = den + torch.exp(sink[hd] - mx)
        out[hd] = e / den
    return out


def talk(weights: torch.Tensor, t: torch.Tensor) -> torch.Tensor:
    return torch.einsum("hg,gij->hij", t, weights)


def attention(h: torch.Tensor, positions: torch.Tensor, m: dict, w: W, p: str, eps: float, **kw) -> torch.Tensor:
    T, H, G, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["vdim"])
    q, k, v = attention_qkv(h, positions, m, w, p, eps)
    pool = int(m["mask"]["pool"])
    a = attention_weights(q, k, pooled_blocks(k, pool), m, w[p + "sink"], **kw)
    a = talk(a, w[p + "talk"])
    values = torch.cat([v, pooled_blocks(v, pool)], 0)
    out = torch.stack([a[hd] @ values[:, hd // (H // G)] for hd in range(H)], 1)
    return out.reshape(T, H * dv) @ w[p + "o"].T


# --------------------------------------------------------------------------------------------------------- time mixing
def wkv_scan(r, k, v, decay, u):
    """r, k, v, decay [T, H, d], u [H, d]: the output reads the state before the token joins it, plus the token's bonus."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=r.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=r.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return out


def wkv_inputs(h: torch.Tensor, m: dict, w: W, p: str):
    T, H, d = h.shape[0], int(m["heads"]), int(m["dim"])
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    mix = {s: h + (prev - h) * w[p + "mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].T).view(T, H, d) for s in "rkv")
    gate = silu(mix["g"] @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(T, H, d)
    return r, k, v, gate, decay


def wkv(h: torch.Tensor, m: dict, w: W, p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    r, k, v, gate, decay = wkv_inputs(h, m, w, p)
    o = rms(wkv_scan(r, k, v, decay, w[p + "u"]), eps).reshape(T, -1)
    return (o * w[p + "norm"] * gate) @ w[p + "o"].T


def parallel(h: torch.Tensor, positions: torch.Tensor, m: dict, w: W, p: str, eps: float) -> torch.Tensor:
    return float(m["left_scale"]) * attention(h, positions, m["left"], w, p + "left.", eps) \
        + float(m["right_scale"]) * wkv(h, m["right"], w, p + "right.", eps)


# -------------------------------------------------------------------------------------------------------------- mamba
def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, inner], A [inner, state], B, C [T, state], D [inner]."""
    S = torch.zeros_like(A)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba1(h: torch.Tensor, m: dict, w: W, p: str) -> torch.Tensor:
    inner, n, rank = int(m["inner"]), int(m["state"]), int(m["dt_rank"])
    xz = h @ w[p + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w[p + "conv"]) + w[p + "conv.b"])
    dbc = x @ w[p + "x"].T
    dt = torch.nn.functional.softplus(dbc[:, :rank] @ w[p + "dt"].T + w[p + "dt.b"], threshold=1e9)
    y = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), dbc[:, rank:rank + n], dbc[:, rank + n:], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------------- feed-forwards
def dense_ff(h: torch.Tensor, mlp: dict, w: W, p: str) -> torch.Tensor:
    limit = float(mlp["limit"])
    g = (h @ w[p + "gate"].T).clamp(max=limit)
    u = (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def gated_ff(h: torch.Tensor, w: W, p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def routing(h: torch.Tensor, mlp: dict, w: W, p: str):
    z = h @ w[p + "router"].T
    top = torch.topk(z, int(mlp["router"]["top"]), dim=-1)
    return top.indices, torch.softmax(top.values, -1)


def moe_ff(h: torch.Tensor, mlp: dict, w: W, p: str) -> torch.Tensor:
    chosen, weight = routing(h, mlp, w, p)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t].tolist(), weight[t]):
            out[t] += c * gated_ff(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + gated_ff(h, w, p + "shared.")
    return out


# ---------------------------------------------------------------------------------------------------------- the model
def layer(x: torch.Tensor, i: int, cfg: dict, w: W) -> torch.Tensor:
    lc, eps, m = cfg["layers"][i], float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    p = f"l{i}."
    positions = torch.arange(x.shape[0])
    h = input_conv(centred_norm(hc_read(x, w, p + "hc1."), w[p + "norm1"], eps), w[p + "canon1"])
    if lc["type"] == "mamba1":
        y = mamba1(h, lc["mixer"], w, p + "mix.")
    elif lc["type"] == "wkv":
        y = wkv(h, lc["mixer"], w, p + "mix.", eps)
    else:
        y = parallel(h, positions, lc["mixer"], w, p + "mix.", eps)
    x = hc_write(x, y, w, p + "hc1.", m)
    if lc.get("mlp") is not None:
        h = centred_norm(hc_read(x, w, p + "hc2."), w[p + "norm2"], eps)
        y = (dense_ff if lc["mlp"]["kind"] == "dense" else moe_ff)(h, lc["mlp"], w, p + "mlp.")
        x = hc_write(x, y, w, p + "hc2.", m)
    return x


def forward(cfg: dict, w: W, tokens: List[int], trace: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; `trace` collects the sum of the streams after every layer."""
    x0 = w["embed"][torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    x = x0[:, None, :].repeat(1, int(cfg["streams"]), 1)
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, w)
        if trace is not None:
            trace.append(x.sum(1))
    return centred_norm(x.sum(1), w["final.norm"], float(cfg["norm"]["eps"])) @ w["embed"].T
