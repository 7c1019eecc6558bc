"""Plain, slow restatement of the Favudra design in torch on the CPU — one function per mechanism, written from the
design's equations and sharing no code with the package.  It takes the config as the plain dict config.json holds and the
weights under their checkpoint names (as float tensors).

Favudra: a residual stream x [T, width] that starts as the scaled embedding; every layer is  x += N_b(mixer(N_a(x)))  then
x += N_d(ff(N_c(x)))  with zero-centred RMS norms N(v) = v / rms(v) * (1 + w).  Mixers: a causal softmax attention whose
q, k, v pass short causal convolutions, with per-head query / key norms, interleaved rotary pairs, tanh-capped scores and a
sink in the softmax's denominator, optionally reading the keys and values an earlier layer cached; gated linear attention
with a decay per key channel; or a windowed attention whose values are its keys, with a linear distance bias per head.  The
feed-forward is SwiGLU; the logits are multiplied by a constant.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F


# --------------------------------------------------------------------------------------------------------------- norms
def rms_norm(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * w


def centred_norm(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_norm(v, 1.0 + w, eps)


# --------------------------------------------------------------------------------------------------- pieces of attention
def short_conv(x: torch.Tensor, taps: torch.Tensor, before: Optional[torch.Tensor]):
    """x [T, C], taps [C, n] (last column meets the current token), before [n − 1, C] or None (zeros) → (y [T, C], the last
    n − 1 inputs)."""
    n = taps.shape[1]
    if before is None:
        before = torch.zeros(n - 1, x.shape[1], dtype=x.dtype)
    full = torch.cat([before, x], 0)
    y = torch.zeros_like(x)
    for j in range(n):
        y = y + taps[:, j] * full[j:j + x.shape[0]]
    return y, full[full.shape[0] - (n - 1):]


def rotate_pairs(v: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """v [T, heads, n]: entries 2i and 2i + 1 of the first rot.dims turn by position · base^(−2i/dims)."""
    if not rot or int(rot["dims"]) == 0:
        return v
    dims = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(v.dtype)[:, None, :], torch.sin(ang).to(v.dtype)[:, None, :]
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out = v.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = a * c - b * s, b * c + a * s
    return out


def capped(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap > 0 else s


def softmax_weights(s: torch.Tensor, visible: torch.Tensor, sink: bool) -> torch.Tensor:
    """Softmax over the visible entries of the last axis; with the sink, 1 joins the denominator."""
    s = s.masked_fill(~visible, float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink:
        top = top.clamp_min(0.0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + (torch.exp(-top) if sink else 0.0))


def distance(pos_q: torch.Tensor, pos_k: torch.Tensor) -> torch.Tensor:
    return pos_q[:, None] - pos_k[None, :]


# ------------------------------------------------------------------------------------------------------ mixer: attention
def attention_keys_values(h, positions, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, mem: dict):
    """The keys [T, kv_heads, dim] (convolved, normed, rotated) and values [T, kv_heads, vdim] (convolved) a layer with
    projections of its own caches; the convolutions' last inputs move on in mem."""
    T, G = h.shape[0], int(m["kv_heads"])
    k, mem["k.in"] = short_conv(h @ w[p + "mix.k"].T, w[p + "mix.k.conv"], mem.get("k.in"))
    v, mem["v.in"] = short_conv(h @ w[p + "mix.v"].T, w[p + "mix.v.conv"], mem.get("v.in"))
    k = rms_norm(k.view(T, G, int(m["dim"])), w[p + "mix.k.norm"], eps)
    return rotate_pairs(k, positions, m.get("rot")), v.view(T, G, int(m["vdim"]))


def attention(h, positions, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, mem: dict, keys, values, key_positions,
              sink: bool = True):
    T, H, G, dk, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, mem["q.in"] = short_conv(h @ w[p + "mix.q"].T, w[p + "mix.q.conv"], mem.get("q.in"))
    q = rotate_pairs(rms_norm(q.view(T, H, dk), w[p + "mix.q.norm"], eps), positions, m.get("rot"))
    visible = distance(positions, key_positions) >= 0
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = capped((q[:, hd] @ keys[:, g].T) * float(m["scale"]), float(m.get("softcap") or 0.0))
        out[:, hd] = softmax_weights(s, visible, sink) @ values[:, g]
    return out.reshape(T, H * dv) @ w[p + "mix.o"].T


# ---------------------------------------------------------------------------------------------------- mixer: attention_2
def slopes(heads: int) -> List[float]:
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def biased_attention(h, positions, m: dict, w: Dict[str, torch.Tensor], p: str, keys, key_positions, bias: bool = True):
    """Windowed attention over keys that are also the values; slope · distance is taken off every score."""
    T, H, G, d = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (h @ w[p + "mix.q"].T).view(T, H, d)
    dist = distance(positions, key_positions)
    size = int((m.get("mask") or {}).get("size", 0))
    visible = (dist >= 0) & ((dist < size) if size > 0 else torch.ones_like(dist, dtype=torch.bool))
    out = torch.zeros(T, H, d, dtype=h.dtype)
    for hd, slope in enumerate(slopes(H)):
        g = hd // (H // G)
        s = (q[:, hd] @ keys[:, g].T) * float(m["scale"])
        if bias:
            s = s - slope * dist.to(h.dtype)
        out[:, hd] = softmax_weights(s, visible, False) @ keys[:, g]
    return out.reshape(T, H * d) @ w[p + "mix.o"].T


# ------------------------------------------------------------------------------------------- mixer: gated linear attention
def gla_mixer(h, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, S: Optional[torch.Tensor]):
    """Token by token: S ← diag(alpha) S + k vᵀ, o = Sᵀ q → (output [T, width], the state [heads, dim, vdim])."""
    T, H, dk, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "mix.q"].T).view(T, H, dk) * dk ** -0.5
    k, v = (h @ w[p + "mix.k"].T).view(T, H, dk), (h @ w[p + "mix.v"].T).view(T, H, dv)
    z = h @ w[p + "mix.a1"].T @ w[p + "mix.a2"].T + w[p + "mix.a2.b"]
    alpha = torch.exp(F.logsigmoid(z) / float(m["tau"])).view(T, H, dk)
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if S is None else S
    o = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o.append((S * q[t][:, :, None]).sum(1))
    o = rms_norm(torch.stack(o), w[p + "mix.norm"], eps).reshape(T, H * dv)
    return (o * F.silu(h @ w[p + "mix.g"].T)) @ w[p + "mix.o"].T, S


# --------------------------------------------------------------------------------------------------------- whole model
def swiglu(h, w: Dict[str, torch.Tensor], p: str):
    return (F.silu(h @ w[p + "mlp.gate"].T) * (h @ w[p + "mlp.up"].T)) @ w[p + "mlp.down"].T


class Sequence:
    """One sequence's memory: what every layer keeps between calls (rows of keys / values, convolution inputs, states)."""

    def __init__(self, cfg: dict):
        self.n = 0
        self.mem: List[dict] = [{} for _ in cfg["layers"]]


def _append(mem: dict, name: str, rows: torch.Tensor):
    mem[name] = torch.cat([mem[name], rows], 0) if name in mem else rows


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, seq: Optional[Sequence] = None, layer_outputs: Optional[list] = None,
            sink: bool = True, bias: bool = True):
    """Logits [T, vocab] of the new tokens of one sequence; `seq` carries the memory of the earlier ones."""
    seq = seq if seq is not None else Sequence(cfg)
    eps = float(cfg["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    T = ids.shape[0]
    positions = torch.arange(seq.n, seq.n + T)
    seen = torch.arange(seq.n + T)
    x = w["embed"][ids] * float(cfg["embedding"]["scale"])
    for i, lc in enumerate(cfg["layers"]):
        p, m, mem = f"l{i}.", lc["mixer"], seq.mem[i]
        h = centred_norm(x, w[p + "norm1"], eps)
        if lc["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                k, v = attention_keys_values(h, positions, m, w, p, eps, mem)
                _append(mem, "k", k), _append(mem, "v", v)
            keep = mem if src is None else seq.mem[int(src)]
            y = attention(h, positions, m, w, p, eps, mem, keep["k"], keep["v"], seen, sink=sink)
        elif lc["type"] == "attention_2":
            _append(mem, "k", (h @ w[p + "mix.k"].T).view(T, int(m["kv_heads"]), int(m["dim"])))
            y = biased_attention(h, positions, m, w, p, mem["k"], seen, bias=bias)
        elif lc["type"] == "gla":
            y, mem["S"] = gla_mixer(h, m, w, p, eps, mem.get("S"))
        else:
            raise ValueError(lc["type"])
        x = x + centred_norm(y, w[p + "norm1b"], eps)
        if lc.get("mlp") is not None:
            x = x + centred_norm(swiglu(centred_norm(x, w[p + "norm2"], eps), w, p), w[p + "norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    seq.n += T
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T * float(cfg["logit_scale"])


def greedy(cfg: dict, w: Dict[str, torch.Tensor], prompt, steps: int) -> List[int]:
    seq = Sequence(cfg)
    out, z = [], forward(cfg, w, prompt, seq)
    for _ in range(steps):
        out.append(int(z[-1].argmax()))
        z = forward(cfg, w, [out[-1]], seq)
    return out
