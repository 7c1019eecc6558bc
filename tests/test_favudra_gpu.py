"""Favudra design in the layer-stack engine against the plain restatement in tests/favudra_oracle.py: every mixer alone as a
one-layer model (whole, decoded, in portions), crafted scores far away, at a window's edges, under the sink, at the cap and
under the distance bias, whole prompts, decoding through caches and states, prompts cut into portions down to one and two
tokens, unequal batches, slots given back and used again, long decoding, other sizes and layer orders, the constants shown to
matter, sizes that reach the tensor-core paths, greedy generation through the engine's own entry points."""
import copy
import math

import pytest
import torch

import favudra_oracle as fo
from tinygpt_b200 import engine, models

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
# fp32 engines are held to summation-order noise on EVERY row; bf16 engines round matrices' operands to 8 bits of mantissa
# and are held to the median row and to most rows against the fp32 restatement.
TOL = {torch.float32: 3e-4, torch.bfloat16: 9e-2}


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


def attn(heads=4, kv_heads=2, dim=12, vdim=20, conv=3, rot={"base": 10000.0, "dims": 8}, softcap=2.0, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "softcap": softcap,
         "scale": scale or 1.3 / math.sqrt(dim)}
    if rot:
        m["rot"] = dict(rot)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def tied(heads=4, kv_heads=2, dim=12, window=9, scale=None):
    """The attention whose values are its keys."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or 1.0 / math.sqrt(dim)}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention_2", "mixer": m}


def gla(heads=3, dim=16, vdim=24, tau=8.0, rank=6):
    """`rank` is a size of the tensors: make() hands it to the reader as a tensor's shape."""
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "rank": rank}


def ff(n=48):
    return {"kind": "dense", "ff": n}


def config(layers, width=64, vocab=96, eps=1e-5, embed=3.0, logit=0.7):
    """→ (config.json as a dict, tensor shapes the reader asks for)."""
    out, shapes = [], {}
    for i, (mix, mlp) in enumerate(layers):
        mix = copy.deepcopy(mix)
        if "rank" in mix:
            shapes[f"l{i}.mix.a1"] = (mix.pop("rank"), width)
        out.append(dict(mix, mlp=copy.deepcopy(mlp)))
    return {"architecture": "Favudra", "embedding": {"scale": embed}, "layers": out, "logit_scale": logit, "norm": {"eps": eps},
            "vocab": vocab, "width": width, "shapes": shapes}


def base_config():
    return config([(attn(), ff()), (tied(), ff(40)), (attn(kv_from=0, softcap=5.0), ff()), (gla(), None),
                   (attn(heads=3, kv_heads=3, dim=10, vdim=6, conv=4, rot={"base": 100.0, "dims": 10}), None),
                   (tied(heads=2, kv_heads=1, dim=20, window=5), ff(24)), (gla(heads=2, dim=40, vdim=16, tau=2.0, rank=11), ff()),
                   (attn(heads=6, kv_heads=3, dim=10, vdim=6, conv=2, rot={"base": 100.0, "dims": 10}, kv_from=4), ff())])


def spec_of(cfg):
    return models.favudra_from_config(cfg, shapes=cfg["shapes"])


def make(cfg, dtype, seed=0, max_ctx=160, max_slots=4, weights=None):
    spec = spec_of(cfg).with_ctx(max_ctx, max_slots)
    w = weights if weights is not None else models.synth_favudra_weights(spec, seed=seed)
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


# ------------------------------------------------------------------------------------------- each mechanism alone
ONE_LAYER = {
    "attention": attn(), "attention_full_rotation": attn(rot={"base": 50.0, "dims": 12}),
    "attention_no_rotation_no_groups": attn(heads=3, kv_heads=3, dim=10, vdim=6, rot=None),
    "attention_one_kv_head": attn(heads=6, kv_heads=1, dim=8, vdim=40, rot={"base": 10.0, "dims": 2}),
    "attention_many_heads_on_one": attn(heads=18, kv_heads=1, dim=8, vdim=8, conv=2, rot={"base": 10.0, "dims": 4}),
    "attention_one_tap": attn(conv=1), "attention_two_taps": attn(conv=2), "attention_six_taps": attn(conv=6, softcap=0.6),
    "attention_no_cap": attn(softcap=0.0), "attention_tight_cap": attn(softcap=0.2, scale=2.0),
    "attention_one_head": attn(heads=1, kv_heads=1, dim=4, vdim=1, rot={"base": 10.0, "dims": 4}),
    "tied": tied(), "tied_no_window": tied(window=0), "tied_no_groups": tied(heads=5, kv_heads=5, dim=7, window=4),
    "tied_one_head": tied(heads=1, kv_heads=1, dim=33, window=2), "tied_window_of_one": tied(window=1),
    "tied_many_heads": tied(heads=12, kv_heads=3, dim=16, window=20),
    "gla": gla(), "gla_one_head": gla(heads=1, dim=8, vdim=8, tau=1.0, rank=1), "gla_wide_key": gla(heads=2, dim=130, vdim=5, rank=3),
    "gla_wide_value": gla(heads=2, dim=5, vdim=700, tau=16.0, rank=9), "gla_square": gla(heads=4, dim=32, vdim=32, tau=4.0, rank=16),
    "gla_longer_key_than_a_slice": gla(heads=1, dim=200, vdim=300, tau=4.0, rank=20),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_one_mixer_alone_whole_decoded_and_in_portions(dtype, name):
    """A model of ONE layer without a feed-forward: the mixer's own path from the stream to the stream — in one go, with a
    decoded tail (caches, states and the convolutions' last inputs carried token by token), in portions of two and one."""
    cfg = config([(ONE_LAYER[name], None)])
    eng, w = make(cfg, dtype)
    toks = tokens(41, cfg["vocab"], 7)
    want = fo.forward(cfg, w, toks)
    for what, got in zip(("whole", "decoded tail", "portions"), run_ways(eng, toks, 30)):
        assert_close(got, want, dtype, what)


def _aim(f, cfg, layer, hk, hq, keys=True, c=10.0):
    """Query rows of `layer` that find the key of ONE normed embedding hk from another, hq: in every head one entry of the key
    is large for hk and the same entry of the query for hq."""
    m, p = cfg["layers"][layer]["mixer"], f"l{layer}.mix."
    dk, last = m["dim"], m["dim"] - 1               # the head's last entry: behind the rotated ones
    assert (m.get("rot") or {"dims": 0})["dims"] < dk
    if keys:
        for g in range(m["kv_heads"]):
            f[p + "k"][g * dk + last] = c * hk / hk.pow(2).sum()
    for h in range(m["heads"]):
        f[p + "q"][h * dk + last] = c * hq / hq.pow(2).sum()
    for nm in ("q", "k"):                           # only the current token's tap: the aim stays on one position
        if p + nm + ".conv" in f:
            f[p + nm + ".conv"] *= 0.02
            f[p + nm + ".conv"][:, -1] = 1.0


def aimed(cfg, seed, n, target, c=10.0):
    """A one-layer model and n tokens in which the LAST token's query is aimed at the key of position `target`: token 0 stands
    only at the target, token 1 only at the end."""
    w = models.synth_favudra_weights(spec_of(cfg), seed=seed)
    toks = tokens(n, cfg["vocab"], seed + 1, low=2)
    toks[target], toks[-1] = 0, 1
    f = {k: v.float() for k, v in w.items()}
    eps, emb = cfg["norm"]["eps"], cfg["embedding"]["scale"]
    hk, hq = (fo.centred_norm(f["embed"][i] * emb, f["l0.norm1"], eps) for i in (0, 1))
    _aim(f, cfg, 0, hk, hq, c=c)
    return {k: v.to(torch.bfloat16) for k, v in f.items()}, toks


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("case", ["last_inside", "first_outside", "far"])
@pytest.mark.parametrize("dim,heads,kv_heads", [(12, 4, 2), (64, 4, 2), (96, 2, 2), (128, 2, 1), (48, 2, 1)])
def test_crafted_scores_at_the_window_edge_and_far_away(dtype, decode, case, dim, heads, kv_heads):
    """300 positions.  The last query is aimed at ONE earlier key so that its score would dominate (the distance bias costs at
    most a few dozen units): the key just inside the window must own the output, the key just outside must not be seen at all,
    and without a window a key 296 positions back must be found — in a prompt and when the last token is decoded alone; also at
    head sizes that send the bf16 engine's prompts to the tensor-core attention kernel and its decode steps to the split-key
    kernels."""
    n, window = 300, 150 if dim == 64 else 61
    cfg = config([(tied(heads, kv_heads, dim, 0 if case == "far" else window, scale=4.0), None)])
    target = {"last_inside": n - window, "first_outside": n - 1 - window, "far": 3}[case]
    w, toks = aimed(cfg, 2, n, target)
    eng, wf = make(cfg, dtype, max_ctx=320, weights=w)
    want = fo.forward(cfg, wf, toks)
    # what the last row would be with a window one key wider (or narrower) tells the cases apart by a wide margin
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["mask"] = {"size": {"last_inside": window - 1, "first_outside": window + 1, "far": 200}[case]}
    assert float(row_err(fo.forward(other, wf, toks)[-1:], want[-1:]).max()) > 0.2
    if decode:
        eng.step([(1, toks[:-1], [])])
        got = eng.step([(1, toks[-1:], [0])])
    else:
        got = eng.step([(1, toks, [n - 1])])
    assert float(row_err(got, want[-1:]).max()) < (1e-4 if dtype == torch.float32 else 6e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dim,vdim", [(12, 20), (64, 64), (96, 96), (128, 128)])
def test_crafted_far_key_of_the_capped_attention_and_of_a_layer_that_shares_it(dtype, decode, dim, vdim):
    """A key 296 positions back, found by a query whose score stands out under the cap; then the same key found by the NEXT
    layer, which has only queries of its own (its input is the first layer's output, so it is aimed along that row)."""
    n, target = 300, 3
    a = dict(heads=4, kv_heads=2, dim=dim, vdim=vdim, rot={"base": 100.0, "dims": dim // 2}, softcap=30.0, scale=1.8 if dim == 12 else 0.6, conv=3)
    for layers in ([(attn(**a), None)], [(attn(**a), None), (attn(kv_from=0, **a), None)]):
        cfg = config(layers)
        w, toks = aimed(cfg, 4, n, target, c=3.0)
        if len(layers) == 2:
            f = {k: v.float() for k, v in w.items()}
            rows = []
            one = dict(cfg, layers=cfg["layers"][:1])
            fo.forward(one, f, toks, layer_outputs=rows)
            f["l1.mix.q"][:] *= 0.2
            _aim(f, cfg, 1, None, fo.centred_norm(rows[0][-1], f["l1.norm1"], cfg["norm"]["eps"]), keys=False, c=3.0)
            w = {k: v.to(torch.bfloat16) for k, v in f.items()}
        eng, wf = make(cfg, dtype, max_ctx=320, weights=w)
        want = fo.forward(cfg, wf, toks)
        blind = list(toks)
        blind[target] = 5
        assert float(row_err(fo.forward(cfg, wf, blind)[-1:], want[-1:]).max()) > 0.2
        if decode:
            eng.step([(1, toks[:-1], [])])
            got = eng.step([(1, toks[-1:], [0])])
        else:
            got = eng.step([(1, toks, [n - 1])])
        assert float(row_err(got, want[-1:]).max()) < (1e-4 if dtype == torch.float32 else 6e-2), len(layers)
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dim,cap", [(12, 0.0), (12, 8.0), (64, 8.0)])
def test_sink_takes_the_weight_when_every_score_is_low(dtype, decode, dim, cap):
    """Head norms with weights of opposite sign on one entry that every token shares: all scores are far below zero, so the sink
    owns the softmax and the heads' outputs vanish; an ordinary softmax would average the values instead."""
    cfg = config([(attn(dim=dim, vdim=dim, rot={"base": 100.0, "dims": 4}, scale=1.0, conv=2, softcap=cap), None)])
    w = models.synth_favudra_weights(spec_of(cfg), seed=4)
    w["embed"][:, 0] = 6.0            # one entry all tokens share …
    for nm, sign in (("q", 1.0), ("k", 1.0)):
        w[f"l0.mix.{nm}"][dim - 1::dim] = 0.0
        w[f"l0.mix.{nm}"][dim - 1::dim, 0] = 4.0     # … lands in the last entry of every head
        w[f"l0.mix.{nm}.conv"][dim - 1::dim] = torch.tensor([0.0, 1.0], dtype=torch.bfloat16)
    w["l0.mix.q.norm"][dim - 1], w["l0.mix.k.norm"][dim - 1] = -3.0, 3.0
    eng, wf = make(cfg, dtype, weights=w)
    toks = tokens(70, cfg["vocab"], 5)
    want = fo.forward(cfg, wf, toks)
    assert float(row_err(fo.forward(cfg, wf, toks, sink=False), want).median()) > 0.2
    got = torch.cat([eng.step([(0, toks[:40], list(range(40)))])] + [eng.step([(0, [t], [0])]) for t in toks[40:]]) if decode \
        else eng.step([(0, toks, list(range(70)))])
    assert_close(got, want, dtype, "sink")


def test_sink_and_distance_bias_matter_with_ordinary_scores():
    cfg = base_config()
    eng, w = make(cfg, torch.float32)
    toks = tokens(30, cfg["vocab"], 6)
    got = eng.step([(0, toks, list(range(30)))])
    assert float(row_err(fo.forward(cfg, w, toks, sink=False), got).max()) > 1e-2
    assert float(row_err(fo.forward(cfg, w, toks, bias=False), got).max()) > 1e-2
    assert_close(got, fo.forward(cfg, w, toks), torch.float32, "with both")


@pytest.mark.parametrize("dtype", DTYPES)
def test_distance_bias_is_the_distance_not_the_position(dtype):
    """The same keys at distances that grow: a bias that used the position, or a slope of the wrong head, would show; 12 heads
    give slopes that are not powers of a half."""
    cfg = config([(tied(heads=12, kv_heads=2, dim=64, window=0, scale=0.02), None)])
    eng, w = make(cfg, dtype, max_ctx=320)
    toks = [7] * 250 + tokens(50, cfg["vocab"], 1)
    want = fo.forward(cfg, w, toks)
    assert float(row_err(fo.forward(cfg, w, toks, bias=False), want)[-1]) > 0.05
    assert_close(eng.step([(0, toks, list(range(300)))]), want, dtype, "whole")
    got = torch.cat([eng.step([(1, toks[:270], list(range(270)))])] + [eng.step([(1, [t], [0])]) for t in toks[270:]])
    assert_close(got, want, dtype, "decoded")


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_linear_attention_keeps_a_value_written_long_ago(dtype):
    """Decays close to one: what the first tokens wrote still shows 200 tokens later (a state that was lost or reset on
    the way would not), whole and with the tail decoded one token at a time."""
    cfg = config([(gla(heads=2, dim=16, vdim=12, tau=64.0), None)])
    w = models.synth_favudra_weights(spec_of(cfg), seed=8)
    w["l0.mix.a2.b"][:] = 6.0
    eng, wf = make(cfg, dtype, max_ctx=256, weights=w)
    toks = tokens(220, cfg["vocab"], 9)
    want = fo.forward(cfg, wf, toks)
    changed = list(toks)
    changed[2] = (toks[2] + 1) % cfg["vocab"]
    assert float(row_err(fo.forward(cfg, wf, changed)[-1:], want[-1:]).max()) > 1e-2
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
    want = fo.forward(cfg, w, toks)
    assert_close(got, want, dtype, "whole prompt")
    assert_close(got[:3], want[:3], dtype, "first tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_then_token_by_token_and_long_decode(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    toks = tokens(120, cfg["vocab"], 8)
    want = fo.forward(cfg, w, toks)
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
    assert_close(torch.cat(rows), fo.forward(cfg, w, toks), dtype, "one by one")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2, 2, 2, 44], [33, 2, 15], [1, 48, 1], [17, 16, 17], [5, 4, 9, 8, 7, 10, 7], [2] * 25])
def test_prompt_in_portions(dtype, cuts):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    toks = tokens(sum(cuts), cfg["vocab"], 10)
    rows, at = [], 0
    for c in cuts:
        rows.append(eng.step([(0, toks[at:at + c], list(range(c)))]))
        at += c
    assert_close(torch.cat(rows), fo.forward(cfg, w, toks), dtype, f"portions {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_against_each_alone_then_decoded_together(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    lens, new = [1, 37, 9], 12
    seqs = [tokens(n + new, cfg["vocab"], 20 + i) for i, n in enumerate(lens)]
    want = [fo.forward(cfg, w, s) for s in seqs]
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
def test_twenty_sequences_decoded_together(dtype):
    """More rows than the batched GEMV and the split-key kernels take."""
    cfg = base_config()
    eng, w = make(cfg, dtype, max_ctx=64, max_slots=20)
    seqs = [tokens(3 + i + 4, cfg["vocab"], 50 + i) for i in range(20)]
    want = [fo.forward(cfg, w, s) for s in seqs]
    eng.step([(i, s[:-4], []) for i, s in enumerate(seqs)])
    for t in range(4):
        got = eng.step([(i, [s[len(s) - 4 + t]], [0]) for i, s in enumerate(seqs)])
        assert_close(got, torch.stack([z[len(z) - 4 + t] for z in want]), dtype, f"step {t}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_prompt_beside_decoding_sequences(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    a, b = tokens(40, cfg["vocab"], 60), tokens(33, cfg["vocab"], 61)
    wa, wb = fo.forward(cfg, w, a), fo.forward(cfg, w, b)
    eng.step([(0, a[:38], [])])
    got = eng.step([(0, [a[38]], [0]), (2, b[:20], list(range(20)))])
    assert_close(got, torch.cat([wa[38:39], wb[:20]]), dtype, "decode token before a prompt")
    got = eng.step([(2, b[20:33], list(range(13))), (0, [a[39]], [0])])
    assert_close(got, torch.cat([wb[20:], wa[39:]]), dtype, "portion before a decode token")


@pytest.mark.parametrize("dtype", DTYPES)
def test_slot_given_back_and_used_again(dtype):
    """A finished request's slot is taken by a new one at position 0: nothing of the old caches, states or convolution
    inputs may show, whether the new request starts with a prompt or with a single token."""
    cfg = base_config()
    eng, w = make(cfg, dtype)
    old = tokens(60, cfg["vocab"], 30)
    eng.step([(1, old, [])])
    for start in (9, 2, 1):
        eng.release(1)
        new = tokens(25, cfg["vocab"], 31 + start)
        rows = [eng.step([(1, new[:start], list(range(start)))])] + [eng.step([(1, [t], [0])]) for t in new[start:]]
        assert_close(torch.cat(rows), fo.forward(cfg, w, new), dtype, f"reused slot, start {start}")


OTHER = {
    "recurrent_first_no_feed_forward_anywhere": [(gla(), None), (attn(), None), (tied(), None)],
    "shared_keys_twice": [(attn(), ff()), (attn(kv_from=0), ff(8)), (tied(), None), (attn(heads=2, kv_from=0, conv=1, softcap=0.0), ff())],
    "two_sources": [(attn(), None), (attn(heads=2, kv_heads=1, dim=8, vdim=8, rot=None), ff()),
                    (attn(heads=2, kv_heads=1, dim=8, vdim=8, rot=None, kv_from=1), ff()), (attn(kv_from=0), None)],
    "one_head_each": [(gla(heads=1, dim=8, vdim=8, tau=1.0, rank=8), None), (tied(heads=1, kv_heads=1, dim=8), None),
                      (attn(heads=1, kv_heads=1, dim=8, vdim=8, conv=1, rot={"base": 10.0, "dims": 8}), ff(16))],
    "odd_sizes": [(attn(heads=3, kv_heads=1, dim=7, vdim=5, conv=5, rot={"base": 7.0, "dims": 6}), ff(13)), (tied(heads=3, kv_heads=3, dim=5, window=6), ff(9)),
                  (gla(heads=3, dim=3, vdim=7, tau=3.0, rank=2), ff(11)), (attn(heads=6, kv_heads=1, dim=7, vdim=5, kv_from=0, rot={"base": 7.0, "dims": 6}), None)],
    "recurrent_only": [(gla(heads=5, dim=3, vdim=40, rank=33), ff()), (gla(tau=1.0), None)],
    "tied_only": [(tied(window=11), None), (tied(heads=8, kv_heads=1, dim=3, window=0), ff())],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(OTHER))
@pytest.mark.parametrize("width,vocab,embed,logit", [(64, 96, 1.0, 1.0), (50, 77, 7.5, 0.11)])
def test_other_layer_orders_and_sizes(dtype, name, width, vocab, embed, logit):
    cfg = config(OTHER[name], width=width, vocab=vocab, eps=1e-6, embed=embed, logit=logit)
    eng, w = make(cfg, dtype, seed=3)
    toks = tokens(36, vocab, 11)
    want = fo.forward(cfg, w, toks)
    assert_close(eng.step([(0, toks, list(range(36)))]), want, dtype, name)
    rows = [eng.step([(2, toks[:7], list(range(7)))])] + [eng.step([(2, toks[t:t + 2], [0, 1][:len(toks[t:t + 2])])])
                                                         for t in range(7, 36, 2)]
    assert_close(torch.cat(rows), want, dtype, name + " in portions of two")


@pytest.mark.parametrize("what", ["eps", "window", "no_window", "rot_base", "rot_dims", "scale", "tied_scale", "softcap", "tau", "embed", "logit_scale",
                                  "kv_from", "conv_state", "shared_softcap"])
def test_constants_matter(what):
    """Each constant of the config changes the logits (a reader that dropped one would go unnoticed otherwise), and the
    engine follows the restatement under the change."""
    cfg = base_config()
    eng, w = make(cfg, torch.float32)
    toks = tokens(40, cfg["vocab"], 12)
    base = eng.step([(0, toks, list(range(40)))])
    eng.close()
    c2 = copy.deepcopy(cfg)
    L = [lc["mixer"] for lc in c2["layers"]]
    if what == "eps":
        c2["norm"]["eps"] = 0.3
    elif what == "window":
        L[1]["mask"]["size"] += 1
    elif what == "no_window":
        del L[5]["mask"]
    elif what == "rot_base":
        L[0]["rot"]["base"] = L[2]["rot"]["base"] = 300.0
    elif what == "rot_dims":
        L[0]["rot"]["dims"] = L[2]["rot"]["dims"] = 4
    elif what == "scale":
        L[0]["scale"] *= 1.7
    elif what == "tied_scale":
        L[1]["scale"] *= 1.7
    elif what == "softcap":
        L[0]["softcap"] = 0.5
    elif what == "shared_softcap":
        L[2]["softcap"] = 0.5
    elif what == "tau":
        L[3]["tau"] = 1.0
    elif what == "embed":
        c2["embedding"]["scale"] = 0.2
    elif what == "logit_scale":
        c2["logit_scale"] = -2.0
    elif what == "kv_from":          # keys and values of its own instead of layer 0's: the tensors must exist
        del L[2]["kv_from"]
    if what == "kv_from":
        w2 = models.synth_favudra_weights(spec_of(c2), seed=5)
        w2 = {k: (w[k].to(torch.bfloat16) if k in w else v) for k, v in w2.items()}
    else:
        w2 = {k: v.to(torch.bfloat16) for k, v in w.items()}
    if what == "conv_state":         # a tap back reads another token: the convolution reaches over the portion's edge
        toks2 = list(toks)
        toks2[17] = (toks[17] + 1) % cfg["vocab"]
        eng2, wf = make(c2, torch.float32, weights=w2)
        got = torch.cat([eng2.step([(0, toks2[:18], list(range(18)))]), eng2.step([(0, toks2[18:], list(range(22)))])])
        assert float(row_err(got[18:20], base[18:20]).max()) > 1e-3
        assert_close(got, fo.forward(c2, wf, toks2), torch.float32, what)
        return
    eng2, wf = make(c2, torch.float32, weights=w2)
    got = eng2.step([(0, toks, list(range(40)))])
    assert float(row_err(got, base).max()) > 1e-3, what
    assert_close(got, fo.forward(c2, wf, toks), torch.float32, what)


def test_every_small_tensor_matters():
    """Norm weights, head norms, taps, decay bias and bottleneck: changing one changes the logits, and the engine follows."""
    cfg = base_config()
    _, w = make(cfg, torch.float32)
    toks = tokens(24, cfg["vocab"], 13)
    base = fo.forward(cfg, w, toks)
    names = [k for k in w if w[k].dim() == 1 or k.endswith(".conv") or k.endswith(".a1") or k.endswith(".a2")]
    assert len(names) > 40
    for k in names[::3]:
        w2 = dict(w)
        w2[k] = (w[k] + 0.5 * torch.randn(w[k].shape, generator=torch.Generator().manual_seed(1))).to(torch.bfloat16).float()
        eng, wf = make(cfg, torch.float32, max_ctx=32, max_slots=1, weights={n: v.to(torch.bfloat16) for n, v in w2.items()})
        got = eng.step([(0, toks, list(range(24)))])
        assert float(row_err(got, base).max()) > 1e-4, k
        assert_close(got, fo.forward(cfg, wf, toks), torch.float32, k)
        eng.close()


def fast_config(dim=64):
    """Sizes that reach the bf16 engines' fast paths: tcgen05 products (widths on multiples of 8, 64 and up), the tensor-core
    prompt attention for both attentions, split-key decode."""
    rot = {"base": 10000.0, "dims": dim // 2}
    return config([(attn(heads=4, kv_heads=2, dim=dim, vdim=dim, softcap=20.0, rot=rot), ff(256)),
                   (tied(heads=4, kv_heads=4, dim=dim, window=48), ff(200)),
                   (gla(heads=4, dim=32, vdim=64, rank=16), ff(256)),
                   (attn(heads=8, kv_heads=2, dim=dim, vdim=dim, softcap=0.0, rot=rot, kv_from=0), None),
                   (tied(heads=6, kv_heads=2, dim=dim, window=0), ff(128))], width=128, vocab=256)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [64, 96, 128])
def test_fast_path_sizes_whole_portions_and_decoded_beside_another(dtype, dim):
    cfg = fast_config(dim)
    eng, w = make(cfg, dtype, max_ctx=320)
    toks, other = tokens(200, cfg["vocab"], 13), tokens(110, cfg["vocab"], 14)
    want = fo.forward(cfg, w, toks)
    whole = eng.step([(0, toks, list(range(200)))])
    assert_close(whole, want, dtype, "whole")
    rows = [eng.step([(1, toks[:64], list(range(64))), (2, other[:50], [])]), eng.step([(1, toks[64:150], list(range(86)))])]
    for t in range(150, 200):
        rows.append(eng.step([(2, [other[50 + t - 150]], []), (1, [toks[t]], [0])]))
    cut = torch.cat(rows)
    assert_close(cut, want, dtype, "portions + decoded beside another request")
    if dtype == torch.bfloat16:       # the bf16 paths agree with each other far better than with the fp32 restatement
        assert float(row_err(cut, whole.float().cpu()).median()) < 3e-2


@pytest.mark.parametrize("cap", [0.3, 3.0, 50.0])
def test_tensor_core_cap_near_and_far_from_its_limit(cap):
    """Scores well inside the cap, around it and far beyond it take different forms of the same function in the prompt kernel."""
    cfg = config([(attn(heads=2, kv_heads=1, dim=64, vdim=64, softcap=cap, scale=0.6, rot={"base": 100.0, "dims": 16}), None)])
    eng, w = make(cfg, torch.bfloat16, max_ctx=160)
    toks = tokens(150, cfg["vocab"], 15)
    want = fo.forward(cfg, w, toks)
    assert float(row_err(fo.forward(dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], softcap=2 * cap))]), w, toks), want).max()) > 1e-4
    e = row_err(eng.step([(0, toks, list(range(150)))]), want)
    assert float(e.median()) < 2e-2 and float(e.max()) < 6e-2


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_engine(dtype):
    cfg = base_config()
    eng, w = make(cfg, dtype)
    prompt, new = tokens(17, cfg["vocab"], 15), 12
    got = eng.generate_sync(prompt, new).tolist()
    seq = list(prompt)
    for i in range(new):              # the restatement's own greedy continuation; a near-tie may part the two in bf16
        lg = fo.forward(cfg, w, seq)[-1]
        top2 = lg.topk(2).values
        if got[i] != int(lg.argmax()):
            assert dtype == torch.bfloat16 and float(top2[0] - top2[1]) < 0.05 * float(lg.std()), (i, got[i], int(lg.argmax()))
            break
        seq.append(got[i])
    if dtype == torch.float32:
        assert got == fo.greedy(cfg, w, prompt, new)
    prompts = [tokens(n, cfg["vocab"], 16 + n) for n in (3, 21, 8)]
    batch = eng.generate_sync_batch(prompts, 6).tolist()
    for p, g in zip(prompts, batch):
        if dtype == torch.float32:
            assert g[0] == int(fo.forward(cfg, w, p)[-1].argmax())
            assert g == eng.generate_sync(p, 6).tolist()


def test_prompt_longer_than_one_pass_of_the_engine():
    """A step of more rows than the engine takes through its layers at once goes in several passes: the states, the
    convolutions' last inputs and the caches (also the shared ones) carry over the seam, also for a batch whose second
    sequence straddles it."""
    a = dict(heads=2, kv_heads=1, dim=8, vdim=8)
    cfg = config([(gla(heads=2, dim=8, vdim=8), None), (attn(**a), ff(16)), (tied(heads=2, kv_heads=1, dim=8, window=30), None),
                  (attn(kv_from=1, **a), None)], width=32, vocab=64)
    n = 4096 + 300
    eng, w = make(cfg, torch.float32, max_ctx=n + 8, max_slots=2)
    toks = tokens(n, 64, 3)
    want = fo.forward(cfg, w, toks)
    idx = list(range(0, n, 211)) + list(range(4090, 4104)) + [n - 1]
    assert_close(eng.step([(0, toks, idx)]), want[idx], torch.float32, "whole")
    eng.release(0)
    got = eng.step([(1, toks[:2500], [2499]), (0, toks[:3000], [0, 2999])])
    assert_close(got, torch.stack([want[2499], want[0], want[2999]]), torch.float32, "batch over the seam")


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
