"""Bibezen design in the layer-stack engine against the plain restatement in tests/bibezen_oracle.py: every mechanism alone (stand-
alone ops and one-layer models: whole, decoded, in portions), crafted scores at the edges of windows and pooled blocks and far
away, whole prompts, decoding through caches and states, prompts cut into portions down to one and two tokens, unequal batches,
slots given back and used again, long decoding, other sizes and layer orders, the constants shown to matter, sizes that reach
the tensor-core paths, greedy generation through the engine's own entry points."""
import copy
import math

import pytest
import torch

import bibezen_oracle as so
from tinygpt_b200 import engine, models, ops

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
# fp32 engines are held to summation-order noise on EVERY row; bf16 engines round matrices' operands to 8 bits of mantissa
# and are held to the median row and to most rows against the fp32 restatement.
TOL = {torch.float32: 2e-4, torch.bfloat16: 9e-2}


def row_err(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per row: rms of the difference (mean removed) over rms of the wanted row (mean removed)."""
    got, want = got.float().cpu(), want.float().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    c = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / c.pow(2).mean(-1).sqrt().clamp_min(1e-6)


def assert_close(got, want, dtype, what=""):
    e = row_err(got, want)
    if dtype == torch.float32:
        assert float(e.max()) < TOL[dtype], f"{what}: worst row {float(e.max()):.2e} at {int(e.argmax())}"
    else:
        assert bool(torch.isfinite(got.float()).all()), what
        assert float(e.median()) < TOL[dtype] and float((e < TOL[dtype]).float().mean()) >= 0.6, \
            f"{what}: {int((e >= TOL[dtype]).sum())} of {len(e)} rows off, median {float(e.median()):.2e}"


def left(heads=4, kv_heads=2, dim=12, vdim=20, window=9, pool=4, conv=3, rot_dims=8, base=100.0, scale=None, softcap=8.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.0 / math.sqrt(dim), "conv": conv,
         "softcap": softcap, "mask": {"size": window, "pool": pool}}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    return m


def wkv(heads=2, dim=16, rank=6):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "rank": rank}}


def parallel(left_scale=0.8, right_scale=0.6, right=None, **kw):
    return {"type": "parallel", "mixer": {"left": left(**kw), "right": dict(right or {"heads": 2, "dim": 8, "rank": 5}),
                                          "left_scale": left_scale, "right_scale": right_scale}}


def mamba(inner=48, state=16, dt_rank=5, conv=4):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}


def ff(n=40, limit=1.2):
    return {"kind": "dense", "ff": n, "limit": limit}


def moe(experts=6, top=2, n=24, shared=32):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": n}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(layers, width=64, vocab=96, eps=1e-5, streams=3, taps=4, mult=0.7, scale=4.0):
    return {"architecture": "Bibezen", "canon": {"taps": taps}, "embedding": {"scale": scale}, "residual_mult": mult, "streams": streams,
            "layers": [dict(copy.deepcopy(mix), mlp=copy.deepcopy(mlp)) for mix, mlp in layers], "norm": {"eps": eps},
            "vocab": vocab, "width": width}


def base_config():
    return config([(parallel(), moe()), (mamba(), ff()), (wkv(), moe(experts=4, top=3, shared=0)), (mamba(inner=40, state=7, dt_rank=9, conv=2), None),
                   (parallel(window=6, pool=3, heads=3, kv_heads=3, dim=10, vdim=9, rot_dims=4, conv=2), ff(24, 0.8))])


def make(cfg, dtype, seed=0, max_ctx=160, max_slots=4, weights=None):
    spec = models.bibezen_from_config(cfg).with_ctx(max_ctx, max_slots)
    w = weights if weights is not None else models.synth_bibezen_weights(spec, seed=seed)
    eng = engine.DecodeEngine(spec, models.pack_weights(spec, w, device=DEV, dtype=dtype))
    return eng, {k: v.float() for k, v in w.items()}


def tokens(n, vocab, seed, low=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(low, vocab, (n,), generator=g).tolist()


def run_ways(eng, toks, head):
    """The same tokens whole, with a decoded tail, and in small portions → three [n, vocab] results."""
    n = len(toks)
    whole = eng.step([(0, toks, list(range(n)))])
    tail = torch.cat([eng.step([(1, toks[:head], list(range(head)))])] + [eng.step([(1, [t], [0])]) for t in toks[head:]])
    rows, at, cuts = [], 0, [2, 1, 2, 2, 1, 1]
    cuts = cuts + [n - sum(cuts) - 2, 2]
    for c in cuts:
        rows.append(eng.step([(3, toks[at:at + c], list(range(c)))]))
        at += c
    return whole, tail, torch.cat(rows)


# ------------------------------------------------------------------------------------------- stand-alone mechanisms
def _i32(*v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams,width,rows", [(1, 40, 3), (2, 64, 200), (3, 50, 7), (4, 1028, 2), (7, 33, 5), (8, 4096, 160)])
def test_hyper_step(dtype, streams, width, rows):
    g = torch.Generator().manual_seed(1)
    x, y = torch.randn(rows, streams, width, generator=g), torch.randn(rows, width, generator=g)
    w = {"p.in": torch.randn(streams, generator=g), "p.out": torch.randn(streams, generator=g), "p.mix": torch.randn(streams, streams, generator=g)}
    nw = 0.2 * torch.randn(width, generator=g)
    want_x = so.hc_write(x, y, w, "p.", 0.6)
    want = so.centred_norm(so.hc_read(want_x, w, "p."), nw, 1e-5)
    d = {k: v.to(DEV).contiguous() for k, v in w.items()}
    xd = x.to(DEV)
    h = ops.stack_hyper_step(xd, d["p.in"], nw.to(DEV), eps=1e-5, y=y.to(DEV), w_out=d["p.out"], mix=d["p.mix"], mult=0.6, dtype=dtype)
    assert float((xd.cpu() - want_x).abs().max()) < 1e-5 * float(want_x.abs().max())
    assert float((h.float().cpu() - want).abs().max()) < (1e-5 if dtype == torch.float32 else 1e-2) * float(want.abs().max())
    h = ops.stack_hyper_step(xd, d["p.in"], nw.to(DEV), eps=1e-5, dtype=dtype)   # without a new output the copies stay
    assert float((xd.cpu() - want_x).abs().max()) < 1e-5 * float(want_x.abs().max())
    assert float((h.float().cpu() - want).abs().max()) < (1e-5 if dtype == torch.float32 else 1e-2) * float(want.abs().max())


@pytest.mark.parametrize("taps", [1, 2, 3, 5])
def test_input_convolution_and_token_shift(taps):
    """Two sequences in one step: one from its start, one that goes on from kept rows."""
    g = torch.Generator().manual_seed(2)
    W, n0, n1, past = 37, 6, 4, 9
    a, b = torch.randn(n0, W, generator=g), torch.randn(past + n1, W, generator=g)
    w, mu = torch.randn(W, taps, generator=g), torch.rand(5, W, generator=g)
    state = torch.full((2, taps, W), 99.0)
    state[1] = b[past - taps:past]
    slot, pos = _i32(*([0] * n0 + [1] * n1)), _i32(*(list(range(n0)) + list(range(past, past + n1))))
    h, mix = ops.stack_input_conv(torch.cat([a, b[past:]]).to(DEV), w.t().contiguous().to(DEV), state.to(DEV), slot, pos, mu=mu.to(DEV))
    ha, hb = so.input_conv(a, w), so.input_conv(b, w)
    prev = torch.cat([torch.zeros(1, W), ha[:-1], hb[past - 1:-1]])
    want = torch.cat([ha, hb[past:]])
    assert float((h.cpu() - want).abs().max()) < 1e-5
    for s in range(5):
        assert float((mix[s].cpu() - (want + (prev - want) * mu[s])).abs().max()) < 1e-5


@pytest.mark.parametrize("dk,dv", [(5, 3), (16, 16), (48, 48), (64, 40), (130, 33)])
def test_bonus_scan_carries_the_state(dk, dv):
    g = torch.Generator().manual_seed(3)
    H, n = 3, 29
    r, k, v = torch.randn(n, H, dk, generator=g), torch.randn(n, H, dk, generator=g), torch.randn(n, H, dv, generator=g)
    decay, u = torch.rand(n, H, dk, generator=g), torch.randn(H, dk, generator=g)
    want = so.wkv_scan(r.double(), k.double(), v.double(), decay.double(), u.double()).reshape(n, H * dv)
    bonus = (r * u * k).sum(-1)
    f = torch.cat([(decay - 1).reshape(n, -1), k.reshape(n, -1), r.reshape(n, -1), v.reshape(n, -1), bonus], 1).to(DEV).contiguous()
    at = [0, H * dk, 2 * H * dk, 3 * H * dk, 3 * H * dk + H * dv, f.shape[1]]
    state = torch.full((2, H * dk * dv), 7.0, device=DEV)
    out, done = [], 0
    for c in (1, 17, 2, 9):
        s = f[done:done + c]
        d_, k_, r_, v_, b_ = (s[:, at[i]:at[i + 1]] for i in range(5))
        out.append(ops.stack_bonus_scan(d_, k_, r_, v_, b_, state, _i32(0), _i32(c), _i32(*([1] * c)), _i32(*range(done, done + c)), heads=H, dk=dk, dv=dv))
        done += c
    e = (torch.cat(out).cpu() - want).abs().max() / want.abs().max()
    assert float(e) < 2e-6 and float((state[0] - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner,n", [(5, 1), (40, 8), (64, 16), (33, 20), (16, 32), (12, 64), (9, 100), (7, 200)])
def test_selective_scan_carries_the_state(dtype, inner, n):
    g = torch.Generator().manual_seed(4)
    T, rank = 75, 3
    x, z = torch.randn(T, inner, generator=g).to(dtype), torch.randn(T, inner, generator=g).to(dtype)
    logit, A_log = torch.randn(T, inner, generator=g) - 1.0, 0.5 * torch.randn(inner, n, generator=g)
    B, C, D = torch.randn(T, n, generator=g), torch.randn(T, n, generator=g), torch.randn(inner, generator=g)
    dt = torch.nn.functional.softplus(logit.double())
    want = so.selective_scan(x.double(), dt, -torch.exp(A_log.double()), B.double(), C.double(), D.double()) * so.silu(z.double())
    xd = torch.cat([torch.zeros(T, 8), B, C, torch.zeros(T, 3)], 1).to(DEV).contiguous()
    state = torch.full((2, inner * n), 3.0, device=DEV)
    out, done = [], 0
    for c in (33, 1, 2, 39):
        s = slice(done, done + c)
        out.append(ops.stack_mamba1_scan(z[s].to(DEV).contiguous(), x[s].to(DEV).contiguous(), xd[s].contiguous(), logit[s].to(DEV).contiguous(), A_log.to(DEV), D.to(DEV),
                                         state, _i32(0), _i32(c), _i32(*([0] * c)), _i32(*range(done, done + c)), dt_rank=rank))
        done += c
    e = (torch.cat(out).double().cpu() - want).abs().max() / want.abs().max()
    assert float(e) < (3e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("splits", [1, 5])
@pytest.mark.parametrize("H,G,dk,dv,size,pool,cap", [(4, 2, 12, 20, 9, 4, 6.0), (3, 3, 7, 5, 5, 1, 0.0), (8, 1, 16, 16, 16, 8, 20.0), (12, 2, 64, 32, 33, 5, 4.0),
                                                      (1, 1, 8, 80, 200, 8, 3.0)])
def test_pool_attention_over_caches(dtype, splits, H, G, dk, dv, size, pool, cap):
    """Prepared queries at every position of a 150-token sequence over cached token and block rows; mixed heads and a sink."""
    g = torch.Generator().manual_seed(5)
    n, ctx = 150, 160
    q, k, v = (torch.randn(n, h, d, generator=g).to(dtype) for h, d in ((H, dk), (G, dk), (G, dv)))
    sink, talk = torch.randn(H, generator=g), torch.eye(H) * 0.7 + 0.3 * torch.randn(H, H, generator=g)
    kc, vc = (torch.zeros(2, ctx + ctx // pool, G * d, dtype=dtype) for d in (dk, dv))
    kb, vb = so.pooled_blocks(k.float(), pool).to(dtype), so.pooled_blocks(v.float(), pool).to(dtype)
    for c, t, b in ((kc, k, kb), (vc, v, vb)):
        c[1, :n] = t.reshape(n, -1)
        c[1, ctx:ctx + n // pool] = b.reshape(n // pool, -1)
    m = {"scale": 0.4, "softcap": cap or 1e9, "mask": {"size": size, "pool": pool}}
    a = so.talk(so.attention_weights(q.double(), k.double(), kb.double(), m, sink.double()), talk.double())
    vals = torch.cat([v, vb], 0).double()
    want = torch.stack([a[h] @ vals[:, h // (H // G)] for h in range(H)], 1).reshape(n, -1)
    got = ops.stack_pool_attention(q.reshape(n, -1).to(DEV), kc.to(DEV), vc.to(DEV), ctx, _i32(*([1] * n)), _i32(*range(n)), heads=H, kv_heads=G, dim=dk,
                                   vdim=dv, scale=0.4, window=size, pool=pool, softcap=cap, sink=sink.to(DEV), talk=talk.to(DEV), splits=splits)
    e = (got.double().cpu() - want).abs().max() / want.abs().max()
    assert float(e) < (3e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [3, 40])
def test_swiglu_experts_with_a_softmax_over_the_chosen(dtype, rows):
    g = torch.Generator().manual_seed(6)
    W, E, F, top = 24, 7, 10, 3
    h = torch.randn(rows, W, generator=g).to(dtype)
    w = {"p.router": torch.randn(E, W, generator=g)}
    for e in range(E):
        w[f"p.e{e}.gate"], w[f"p.e{e}.up"], w[f"p.e{e}.down"] = (torch.randn(*s, generator=g) * 0.4 for s in ((F, W), (F, W), (W, F)))
    w = {k: v.to(dtype).float() for k, v in w.items()}
    w_in = torch.stack([torch.cat([w[f"p.e{e}.gate"], w[f"p.e{e}.up"]]) for e in range(E)]).to(dtype).to(DEV)
    w_out = torch.stack([w[f"p.e{e}.down"] for e in range(E)]).to(dtype).to(DEV)
    y, chosen, weight = ops.stack_moe(h.to(DEV), w["p.router"].to(dtype).to(DEV), w_in, w_out, top, 0.0, chosen_only=True, weight_output=True,
                                      act="glu_silu")
    mlp = {"router": {"top": top}}
    wc, ww = so.routing(h.float(), mlp, w, "p.")
    assert torch.equal(chosen.cpu().long(), wc) and float((weight.cpu() - ww).abs().max()) < 1e-5
    want = so.moe_ff(h.float(), mlp, w, "p.")
    assert float((y.cpu() - want).abs().max() / want.abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2)


# ------------------------------------------------------------------------------------------- one-layer models
ONE_LAYER = {
    "parallel": parallel(), "parallel_pool_of_one": parallel(window=3, pool=1),
    "parallel_no_rotation_no_groups": parallel(heads=3, kv_heads=3, dim=10, vdim=6, window=4, pool=7, rot_dims=0),
    "parallel_one_kv_head_one_tap": parallel(heads=6, kv_heads=1, dim=8, vdim=40, window=13, pool=2, rot_dims=8, conv=1),
    "parallel_one_head_window_of_one": parallel(heads=1, kv_heads=1, dim=4, vdim=33, window=1, pool=3, rot_dims=2, conv=5),
    "parallel_wide_window": parallel(window=64, pool=4), "parallel_odd_right": parallel(right={"heads": 3, "dim": 7, "rank": 17}, vdim=7),
    "wkv": wkv(), "wkv_one_head": wkv(heads=1, dim=40, rank=1), "wkv_odd": wkv(heads=5, dim=9, rank=13), "wkv_wide": wkv(heads=1, dim=70, rank=8),
    "mamba": mamba(), "mamba_one_tap": mamba(inner=30, state=4, dt_rank=1, conv=1), "mamba_odd": mamba(inner=37, state=19, dt_rank=11, conv=6),
    "mamba_wide_state": mamba(inner=24, state=70, dt_rank=8, conv=3),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_one_mixer_alone_whole_decoded_and_in_portions(dtype, name):
    """A model of ONE layer without a feed-forward: the mixer's own path from the copies to the copies — in one go, with a
    decoded tail (caches, states and every convolution's last inputs carried token by token), in portions of two and one."""
    cfg = config([(ONE_LAYER[name], None)])
    eng, w = make(cfg, dtype)
    toks = tokens(41, cfg["vocab"], 7)
    want = so.forward(cfg, w, toks)
    for what, got in zip(("whole", "decoded tail", "portions"), run_ways(eng, toks, 30)):
        assert_close(got, want, dtype, what)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams,taps", [(1, 1), (1, 3), (2, 5), (4, 2), (6, 3)])
def test_streams_and_input_taps(dtype, streams, taps):
    cfg = config([(wkv(), ff()), (mamba(), moe())], streams=streams, taps=taps)
    eng, w = make(cfg, dtype)
    toks = tokens(33, cfg["vocab"], 8)
    want = so.forward(cfg, w, toks)
    for what, got in zip(("whole", "decoded tail", "portions"), run_ways(eng, toks, 20)):
        assert_close(got, want, dtype, what)


def _aimed(cfg, seed, n, targets):
    """A one-layer model and n tokens in which the LAST token's query is aimed at the keys of the target positions: token 0 stands
    only there, token 1 only at the end; every convolution passes the current row alone; in every head the rows of the key
    projection that feed one unrotated entry are set along token 0's input and the query's along token 1's, so that after the
    head norms both vectors are almost that entry alone."""
    spec = models.bibezen_from_config(cfg)
    f = {k: v.float() for k, v in models.synth_bibezen_weights(spec, seed=seed).items()}
    toks = tokens(n, cfg["vocab"], seed + 1, low=2)
    for t in targets:
        toks[t] = 0
    toks[-1] = 1
    m, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    f["l0.canon1"][:] = 0.0
    for s in "qkv":
        f[p + s + ".conv"][:] = 0.0
        f[p + s + ".conv"][:, -1] = 1.0
    u = f["embed"][:2] * cfg["embedding"]["scale"] * f["l0.hc1.in"].sum()
    hk, hq = so.centred_norm(u, f["l0.norm1"], cfg["norm"]["eps"])
    dk, last = m["dim"], m["dim"] - 1
    assert (m.get("rot") or {"dims": 0})["dims"] < dk
    f[p + "q.norm"][:], f[p + "k.norm"][:] = 1.0, 1.0
    for nm, heads, h in (("k", m["kv_heads"], hk), ("q", m["heads"], hq)):
        for i in range(heads):
            f[p + nm][i * dk + last] = 12.0 * h / h.pow(2).sum()
            f[p + nm + ".b"][i * dk + last] = 0.0
    f[p + "sink"][:] = -3.0
    return {k: v.to(torch.bfloat16) for k, v in f.items()}, toks


SIZES = {"any_size": dict(heads=4, kv_heads=2, dim=18, vdim=10, rot_dims=4), "tensor_core_sizes": dict(heads=6, kv_heads=2, dim=32, vdim=48, rot_dims=8),
         "many_heads": dict(heads=20, kv_heads=4, dim=16, vdim=80, rot_dims=2)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("case", ["token_last_inside", "token_first_outside", "block_just_seen", "block_not_yet_seen", "far_block"])
@pytest.mark.parametrize("size", sorted(SIZES))
def test_crafted_scores_at_window_and_block_edges_and_far_away(dtype, decode, case, size):
    """300 positions, a window of 61 and blocks of 4.  The last query is aimed at ONE key: the token just inside the window and a
    whole block that ends just before it must own the output; the token just outside (its block not yet whole before the
    window) and a block that still reaches into the window's edge must not be seen; a block near the start must be found."""
    # the last position is 299.  Window 61: tokens 239 … 299, and the block 236 … 239 ends one position too late.  Window 64: tokens
    # 236 … 299, and the block 232 … 235 ends just before them.
    n, pool, window = 300, 4, 64 if case == "block_just_seen" else 61
    cfg = config([(parallel(window=window, pool=pool, conv=2, softcap=25.0, scale=1.0, left_scale=3.0, right_scale=0.1, **SIZES[size]), None)], streams=2)
    targets = {"token_last_inside": [239], "token_first_outside": [238], "block_just_seen": [232, 233, 234, 235],
               "block_not_yet_seen": [236, 237, 238], "far_block": [4, 5, 6, 7]}[case]
    w, toks = _aimed(cfg, 2, n, targets)
    eng, wf = make(cfg, dtype, max_ctx=320, weights=w)
    want = so.forward(cfg, wf, toks)
    # what the last row would be with another window or without pooled blocks tells the cases apart by a wide margin
    other = copy.deepcopy(cfg)
    mask = other["layers"][0]["mixer"]["left"]["mask"]
    mask.update({"token_last_inside": {"size": window - 1}, "token_first_outside": {"size": window + 1}, "block_just_seen": {"size": window, "pool": 1000},
                 "block_not_yet_seen": {"size": window - 1}, "far_block": {"size": window, "pool": 1000}}[case])
    assert float(row_err(so.forward(other, wf, toks)[-1:], want[-1:]).max()) > 0.1
    if decode:
        eng.step([(1, toks[:-1], [])])
        got = eng.step([(1, toks[-1:], [0])])
    else:
        got = eng.step([(1, toks, [n - 1])])
    assert float(row_err(got, want[-1:]).max()) < (1e-4 if dtype == torch.float32 else 6e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
def test_sink_takes_the_weight_when_every_score_is_low(dtype, decode):
    """Queries and keys point away from each other and the sinks are high: the sinks own the softmax and the attention's share
    of the output almost vanishes; without them it would average the values instead."""
    cfg = config([(parallel(rot_dims=4, scale=1.0, softcap=20.0, right_scale=0.05), None)], streams=2)
    spec = models.bibezen_from_config(cfg)
    w = models.synth_bibezen_weights(spec, seed=4)
    dk, p = cfg["layers"][0]["mixer"]["left"]["dim"], "l0.mix.left."
    for nm, heads, v in (("k", 2, 6.0), ("q", 4, -6.0)):
        for i in range(heads):
            w[p + nm + ".b"][i * dk + dk - 1] = v
        w[p + nm + ".conv"][:, :-1] = 0.0
        w[p + nm + ".conv"][:, -1] = 1.0
    w[p + "sink"][:] = 3.0
    eng, wf = make(cfg, dtype, weights=w)
    toks = tokens(70, cfg["vocab"], 5)
    want = so.forward(cfg, wf, toks)
    low = {k: v.clone() for k, v in wf.items()}
    low[p + "sink"][:] = -60.0
    assert float(row_err(so.forward(cfg, low, toks), want).min()) > 0.1
    got = torch.cat([eng.step([(0, toks[:40], list(range(40)))])] + [eng.step([(0, [t], [0])]) for t in toks[40:]]) if decode \
        else eng.step([(0, toks, list(range(70)))])
    assert_close(got, want, dtype, "sink")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["wkv", "mamba1"])
def test_recurrences_keep_what_was_written_long_ago(dtype, kind):
    """Decays close to one: what the first tokens wrote still shows 200 tokens later (a state that was lost or reset on the way
    would not), whole and with the tail decoded one token at a time."""
    cfg = config([(wkv(heads=2, dim=16) if kind == "wkv" else mamba(inner=32, state=8), None)], streams=2, taps=2)
    spec = models.bibezen_from_config(cfg)
    w = models.synth_bibezen_weights(spec, seed=8)
    if kind == "wkv":
        w["l0.mix.w0"][:] = -8.0
    else:
        w["l0.mix.A_log"][:] = -7.0
        w["l0.mix.x"] = w["l0.mix.x"] * 5.0   # what the state holds weighs more than the token's own share
    eng, wf = make(cfg, dtype, max_ctx=256, weights=w)
    toks = tokens(220, cfg["vocab"], 9)
    want = so.forward(cfg, wf, toks)
    changed = list(toks)
    changed[:8] = [(t + 1) % cfg["vocab"] for t in toks[:8]]
    assert float(row_err(so.forward(cfg, wf, changed)[-1:], want[-1:]).max()) > 3e-3
    got = torch.cat([eng.step([(2, toks[:150], list(range(150)))])] + [eng.step([(2, [t], [0])]) for t in toks[150:]])
    assert_close(got, want, dtype, "long memory")
    assert_close(eng.step([(1, toks, [219])]), want[-1:], dtype, "whole")


# ------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompt(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    toks = tokens(50, cfg["vocab"], 7)
    got = eng.step([(0, toks, list(range(50)))])
    want = so.forward(cfg, w, toks)
    assert_close(got, want, dtype, "whole prompt")
    assert_close(got[:3], want[:3], dtype, "first tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_then_token_by_token_and_long_decode(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    toks = tokens(120, cfg["vocab"], 8)
    want = so.forward(cfg, w, toks)
    rows = [eng.step([(2, toks[:30], list(range(30)))])]
    for t in range(30, 120):
        rows.append(eng.step([(2, [toks[t]], [0])]))
    assert_close(torch.cat(rows), want, dtype, "prefill + 90 decode steps")
    assert eng.slot_position(2) == 120


@pytest.mark.parametrize("dtype", DTYPES)
def test_from_the_first_token_one_by_one(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    toks = tokens(20, cfg["vocab"], 9)
    rows = [eng.step([(1, [t], [0])]) for t in toks]
    assert_close(torch.cat(rows), so.forward(cfg, w, toks), dtype, "one by one")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2, 2, 2, 44], [33, 2, 15], [1, 48, 1], [17, 16, 17], [5, 4, 9, 8, 7, 10, 7]])
def test_prompt_in_portions(dtype, cuts):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    toks = tokens(sum(cuts), cfg["vocab"], 10)
    rows, at = [], 0
    for c in cuts:
        rows.append(eng.step([(0, toks[at:at + c], list(range(c)))]))
        at += c
    assert_close(torch.cat(rows), so.forward(cfg, w, toks), dtype, f"portions {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_against_each_alone_then_decoded_together(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    lens, new = [1, 37, 9], 12
    seqs = [tokens(n + new, cfg["vocab"], 20 + i) for i, n in enumerate(lens)]
    want = [so.forward(cfg, w, s) for s in seqs]
    slots = [3, 0, 2]
    got = eng.step([(sl, s[:n], list(range(n))) for sl, s, n in zip(slots, seqs, lens)])
    at = 0
    for i, n in enumerate(lens):
        assert_close(got[at:at + n], want[i][:n], dtype, f"batched prompt {i}")
        at += n
    live = [0, 1, 2]
    for t in range(new):
        if t == 5:                       # the middle request ends early; its slot goes back
            eng.release(slots[1])
            live = [0, 2]
        got = eng.step([(slots[i], [seqs[i][lens[i] + t]], [0]) for i in live])
        for r, i in enumerate(live):
            assert_close(got[r:r + 1], want[i][lens[i] + t:lens[i] + t + 1], dtype, f"decoded together {i} step {t}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_batches_decode_alike(dtype):
    """24 sequences decoded together (more rows than the small products and the key splits of a single row are made for)."""
    cfg = base_config()
    eng, w = make(cfg, dtype, max_ctx=64, max_slots=24)
    seqs = [tokens(30, cfg["vocab"], 50 + i) for i in range(24)]
    eng.step([(i, s[:5 + i % 7], []) for i, s in enumerate(seqs)])
    for t in range(4):
        got = eng.step([(i, [s[5 + i % 7 + t]], [0]) for i, s in enumerate(seqs)])
    for i in (0, 3, 13, 23):
        n = 5 + i % 7 + 4
        assert_close(got[i:i + 1], so.forward(cfg, w, seqs[i][:n])[-1:], dtype, f"sequence {i}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_slot_given_back_and_used_again(dtype):
    """A finished request's slot is taken by a new one at position 0: nothing of the old caches, pooled blocks, states or
    convolution inputs may show, whether the new request starts with a prompt or with a single token."""
    cfg = base_config()
    eng, w = make(cfg, dtype)
    old = tokens(60, cfg["vocab"], 30)
    eng.step([(1, old, [])])
    for start in (9, 1):
        eng.release(1)
        new = tokens(25, cfg["vocab"], 31 + start)
        rows = [eng.step([(1, new[:start], list(range(start)))])] + [eng.step([(1, [t], [0])]) for t in new[start:]]
        assert_close(torch.cat(rows), so.forward(cfg, w, new), dtype, f"reused slot, start {start}")


OTHER = {
    "recurrences_only": [(wkv(), None), (mamba(), None), (wkv(heads=3, dim=8), ff(8))],
    "attention_twice_then_wkv": [(parallel(window=2, pool=5), None), (parallel(heads=2, kv_heads=1, dim=8, vdim=8, window=20, pool=2, rot_dims=8), moe(shared=0)), (wkv(), None)],
    "equal_sizes": [(parallel(heads=4, kv_heads=4, dim=16, vdim=16, window=8, pool=8, conv=4, rot_dims=16, right={"heads": 4, "dim": 16, "rank": 16}), moe(4, 4, 16, 16)),
                    (mamba(inner=64, state=16, dt_rank=16, conv=4), ff(64, 4.0)), (wkv(heads=4, dim=16, rank=16), moe(4, 1, 16, 16))],
    "all_ones": [(parallel(heads=1, kv_heads=1, dim=2, vdim=1, window=1, pool=1, conv=1, rot_dims=2, right={"heads": 1, "dim": 1, "rank": 1}), moe(1, 1, 1, 1)),
                 (mamba(inner=1, state=1, dt_rank=1, conv=1), ff(1))],
    "many_experts": [(mamba(), moe(40, 5, 8, 8)), (wkv(), moe(3, 3, 8, 0))],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(OTHER))
@pytest.mark.parametrize("width,vocab,streams,taps", [(64, 96, 2, 3), (50, 77, 3, 2)])
def test_other_layer_orders_and_sizes(dtype, name, width, vocab, streams, taps):
    cfg = config(OTHER[name], width=width, vocab=vocab, eps=1e-6, streams=streams, taps=taps, mult=1.0, scale=1.0 if name == "all_ones" else 6.0)
    eng, w = make(cfg, dtype, seed=3)
    toks = tokens(36, vocab, 11)
    want = so.forward(cfg, w, toks)
    assert_close(eng.step([(0, toks, list(range(36)))]), want, dtype, name)
    rows = [eng.step([(2, toks[:7], list(range(7)))])] + [eng.step([(2, toks[t:t + 2], [0, 1][:len(toks[t:t + 2])])])
                                                         for t in range(7, 36, 2)]
    assert_close(torch.cat(rows), want, dtype, name + " in portions of two")


CONSTANTS = {
    "eps": (("norm", "eps"), 0.3), "residual_mult": (("residual_mult",), 1.1), "embedding_scale": (("embedding", "scale"), 0.3),
    "window": ((0, "mixer", "left", "mask", "size"), 10), "pool": ((0, "mixer", "left", "mask", "pool"), 3),
    "scale": ((0, "mixer", "left", "scale"), 0.5), "softcap": ((0, "mixer", "left", "softcap"), 1.0),
    "rot_base": ((0, "mixer", "left", "rot", "base"), 3.0), "rot_dims": ((0, "mixer", "left", "rot", "dims"), 4),
    "left_scale": ((0, "mixer", "left_scale"), 0.2), "right_scale": ((0, "mixer", "right_scale"), 1.5), "limit": ((1, "mlp", "limit"), 0.2),
    "top": ((0, "mlp", "router", "top"), 3),
}


@pytest.mark.parametrize("what", sorted(CONSTANTS))
def test_constants_matter(what):
    """Each constant of the config changes the logits (a reader that dropped one would go unnoticed otherwise), and the
    engine follows the restatement under the change."""
    cfg = base_config()
    spec = models.bibezen_from_config(cfg)
    w = models.synth_bibezen_weights(spec, seed=0)
    for k in w:                         # scores, gates and hidden rows large enough for caps and clamps to bite
        if k.endswith("left.q.norm"):
            w[k] = w[k] * 2.0
        if k == "l1.mlp.gate" or k == "l1.mlp.up":
            w[k] = w[k] * 4.0
    eng, _ = make(cfg, torch.float32, weights=w)
    toks = tokens(40, cfg["vocab"], 12)
    base = eng.step([(0, toks, list(range(40)))])
    eng.close()
    c2 = copy.deepcopy(cfg)
    path, value = CONSTANTS[what]
    node = c2["layers"] if isinstance(path[0], int) else c2
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    eng2, wf = make(c2, torch.float32, weights=w)
    got = eng2.step([(0, toks, list(range(40)))])
    assert float(row_err(got, base).max()) > 1e-3, what
    assert_close(got, so.forward(c2, wf, toks), torch.float32, what)


@pytest.mark.parametrize("tensor", ["left.talk", "left.sink", "left.q.conv", "left.v.conv", "left.q.b", "left.k.norm", "right.u", "right.mu.w", "right.w0",
                                    "right.norm", "canon1", "hc1.in", "hc1.out", "hc1.mix", "hc2.mix"])
def test_every_small_tensor_matters(tensor):
    """Replacing one small tensor by its neutral value changes the logits, and the engine follows: none is left out."""
    cfg = config([(parallel(), ff())])
    spec = models.bibezen_from_config(cfg)
    w = models.synth_bibezen_weights(spec, seed=1)
    toks = tokens(40, cfg["vocab"], 12)
    f = {k: v.float() for k, v in w.items()}
    want = so.forward(cfg, f, toks)
    name = "l0." + ("mix." if tensor[:4] in ("left", "righ") else "") + tensor
    w2 = dict(w)
    w2[name] = torch.zeros_like(w[name]) if tensor not in ("left.talk", "hc1.mix", "hc2.mix") else torch.eye(w[name].shape[0]).to(torch.bfloat16)
    if "conv" in name:
        w2[name][:, -1] = 1.0
    if tensor == "left.sink":
        w2[name] = w[name] - 9.0
    eng, wf = make(cfg, torch.float32, weights=w2)
    got = eng.step([(0, toks, list(range(40)))])
    assert float(row_err(got, want).max()) > 1e-3, tensor
    assert_close(got, so.forward(cfg, wf, toks), torch.float32, tensor)


def fast_config():
    """Sizes that reach the bf16 engines' fast paths: tcgen05 products (multiples of 8, 64 and up) also for the bottlenecks and
    the experts, the tensor-core prompt attention (head sizes on multiples of 16; one and two warps' worth of heads; value
    columns split over CTAs), split-key decode."""
    return config([(parallel(heads=10, kv_heads=5, dim=48, vdim=112, window=40, pool=6, conv=4, rot_dims=32, right={"heads": 4, "dim": 32, "rank": 64}), moe(4, 2, 64, 96)),
                   (mamba(inner=256, state=16, dt_rank=64, conv=4), ff(256)), (wkv(heads=2, dim=64, rank=64), moe(4, 2, 64, 64)),
                   (parallel(heads=24, kv_heads=8, dim=16, vdim=96, window=70, pool=16, rot_dims=16, right={"heads": 2, "dim": 64, "rank": 24}), ff(128)),
                   (parallel(heads=4, kv_heads=2, dim=128, vdim=144, window=33, pool=4, rot_dims=128, right={"heads": 2, "dim": 64, "rank": 24}), None)],
                  width=128, vocab=256, streams=2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_fast_path_sizes_whole_portions_and_decoded_beside_another(dtype):
    cfg = fast_config()
    eng, w = make(cfg, dtype, max_ctx=320)
    toks, other = tokens(200, cfg["vocab"], 13), tokens(110, cfg["vocab"], 14)
    want = so.forward(cfg, w, toks)
    whole = eng.step([(0, toks, list(range(200)))])
    assert_close(whole, want, dtype, "whole")
    rows = [eng.step([(1, toks[:64], list(range(64))), (2, other[:50], [])]), eng.step([(1, toks[64:150], list(range(86)))])]
    for t in range(150, 200):
        rows.append(eng.step([(2, [other[50 + t - 150]], []), (1, [toks[t]], [0])]))
    cut = torch.cat(rows)
    assert_close(cut, want, dtype, "portions + decoded beside another request")
    if dtype == torch.bfloat16:       # the bf16 paths agree with each other far better than with the fp32 restatement
        e = row_err(cut, whole.float().cpu())
        assert float(e.median()) < 3e-2


def test_prompt_longer_than_one_pass_of_the_engine():
    """A step of more rows than the engine takes through its layers at once goes in several passes: states, the convolutions' last
    inputs, caches and pooled blocks carry over the seam, also for a batch whose second sequence straddles it."""
    cfg = config([(parallel(heads=2, kv_heads=1, dim=8, vdim=8, window=40, pool=7, rot_dims=8), None), (wkv(heads=1, dim=8), ff(8)),
                  (mamba(inner=16, state=4), None)], width=32, vocab=64, streams=2)
    n = 4096 + 300
    eng, w = make(cfg, torch.float32, max_ctx=n + 8, max_slots=2)
    toks = tokens(n, 64, 3)
    want = so.forward(cfg, w, toks)
    idx = list(range(0, n, 211)) + list(range(4090, 4104)) + [n - 1]
    assert_close(eng.step([(0, toks, idx)]), want[idx], torch.float32, "whole")
    eng.release(0)
    got = eng.step([(1, toks[:2500], [2499]), (0, toks[:3000], [0, 2999])])
    assert_close(got, torch.stack([want[2499], want[0], want[2999]]), torch.float32, "batch over the seam")


def greedy(cfg, w, prompt, new):
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(so.forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_engine(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    prompt, new = tokens(17, cfg["vocab"], 15), 24
    got = eng.generate_sync(prompt, new).tolist()
    seq = list(prompt)
    for i in range(new):              # the restatement's own greedy continuation; a near-tie may part the two in bf16
        lg = so.forward(cfg, w, seq)[-1]
        top2 = lg.topk(2).values
        if got[i] != int(lg.argmax()):
            assert dtype == torch.bfloat16 and float(top2[0] - top2[1]) < 0.08 * float(lg.std()), (i, got[i], int(lg.argmax()))
            break
        seq.append(got[i])
    prompts = [tokens(n, cfg["vocab"], 16 + n) for n in (3, 21, 8)]
    batch = eng.generate_ragged(prompts, 6)
    if dtype == torch.float32:
        assert got == greedy(cfg, w, prompt, new)
        assert batch == [greedy(cfg, w, p, 6) for p in prompts]


def test_seek_and_overflow_refused():
    cfg = base_config()
    eng, _ = make(cfg, torch.float32, max_ctx=32)
    toks = tokens(20, cfg["vocab"], 17)
    eng.step([(0, toks, [])], greedy=True)
    with pytest.raises(Exception):
        eng.seek(5)                   # the recurrent states hold the whole prefix and nothing of its past
    with pytest.raises(Exception):
        eng.step([(0, toks, [])])     # 20 + 20 > 32
    assert eng.slot_position(0) == 20
