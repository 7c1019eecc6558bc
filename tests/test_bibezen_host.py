"""Host side of the Bibezen design (no GPU): config reader and registry, merged layouts, packed weights, checkpoint round trip
through the loader (the bottleneck's rank comes from the tensors), and the restatement's own sanity — causality, closed forms
of the connections, the convolutions, the pooled blocks, the mixed heads and the recurrences."""
import copy

import pytest
import torch

import bibezen_oracle as so
from tinygpt_b200 import loader, models


def cfg_small():
    return {"architecture": "Bibezen", "width": 40, "vocab": 50, "norm": {"eps": 1e-4}, "canon": {"taps": 4}, "embedding": {"scale": 3.0},
            "residual_mult": 0.6, "streams": 3,
            "layers": [
                {"type": "parallel", "mixer": {
                    "left": {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 6, "scale": 0.3, "conv": 2, "softcap": 9.0,
                             "mask": {"size": 5, "pool": 3}, "rot": {"base": 50.0, "dims": 6}},
                    "left_scale": 0.7, "right": {"heads": 2, "dim": 9}, "right_scale": 0.4}, "mlp": {"kind": "dense", "ff": 24, "limit": 1.5}},
                {"type": "mamba1", "mixer": {"inner": 22, "state": 5, "dt_rank": 3, "conv": 3}, "mlp": None},
                {"type": "wkv", "mixer": {"heads": 3, "dim": 7},
                 "mlp": {"kind": "moe", "router": {"experts": 5, "top": 2}, "expert": {"ff": 12}, "shared": {"ff": 20}}},
                {"type": "mamba1", "mixer": {"inner": 16, "state": 4, "dt_rank": 9, "conv": 1},
                 "mlp": {"kind": "moe", "router": {"experts": 3, "top": 3}, "expert": {"ff": 8}}}]}


def test_registry_reads_the_config_and_writes_it_back():
    cfg = cfg_small()
    spec = models.ARCHITECTURES["Bibezen"](cfg)
    assert spec.block == "hyper" and spec.streams == 3 and spec.norm_offset == 1.0 and spec.norm_kind == "rms"
    assert spec.embed_scale == 3.0 and spec.residual_mult == 0.6 and spec.norm_eps == 1e-4 and [r[0] for r in spec.runs()] == [0, 1, 2, 3]
    L = spec.layers[0]
    a = L.pool
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.conv, a.window, a.pool, a.softcap, a.scale) == (4, 2, 10, 6, 2, 5, 3, 9.0, 0.3)
    assert a.rot.dims == 6 and a.rot.base == 50.0 and (L.left_scale, L.right_scale) == (0.7, 0.4) and L.canon == 4
    assert (L.wkv.heads, L.wkv.dim) == (2, 9) and L.ff_kind == "glu_clamp" and (L.ff, L.ff_limit) == (24, 1.5)
    m = spec.layers[1].mamba1
    assert (m.inner, m.state, m.dt_rank, m.conv) == (22, 5, 3, 3) and spec.layers[1].ff == 0
    q = spec.layers[2].moe
    assert (q.experts, q.top, q.expert_ff, q.shared_ff, q.router, q.act) == (5, 2, 12, 20, "softmax_chosen", "glu_silu")
    assert spec.layers[3].moe.shared_ff == 0
    assert models.bibezen_config(spec) == cfg and models.bibezen_from_config(models.bibezen_config(spec)) == spec


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "latent"), (("layers", 0, "mlp", "kind"), "gelu"), (("layers", 0, "mixer", "left", "kv_heads"), 3),
    (("layers", 0, "mixer", "left", "rot", "dims"), 12), (("layers", 0, "mixer", "left", "rot", "dims"), 5),
    (("layers", 0, "mixer", "left", "conv"), 0), (("layers", 1, "mixer", "state"), 0), (("layers", 2, "mlp", "router", "top"), 6),
    (("streams",), 0)])
def test_configs_outside_the_design_are_refused(path, value):
    cfg = cfg_small()
    node = cfg
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(ValueError):
        models.bibezen_from_config(cfg)


def test_visibility_of_the_spec_and_of_the_restatement_agree():
    a = models.bibezen_from_config(cfg_small()).layers[0].pool
    n = 40
    tok, blk = so.visible_tokens(n, 5), so.visible_blocks(n, n // 3, 3, 5)
    for i in range(n):
        assert [a.visible(i, j) for j in range(n)] == tok[i].tolist()
        assert [a.visible_block(i, b) for b in range(n // 3)] == blk[i].tolist()
    assert bool(blk[7, 0]) and not bool(blk[6, 0]) and not bool(blk[9, 1]) and bool(blk[10, 1])


def test_packed_weights_lie_where_the_layout_says():
    spec = models.bibezen_from_config(cfg_small())
    w = models.synth_bibezen_weights(spec, seed=1)
    p = models.pack_weights(spec, w, device="cpu")
    lay = spec.mix_layout(0)
    assert lay.off_q % 8 == lay.off_k % 8 == lay.off_v % 8 == lay.k_out % 8 == 0
    assert torch.equal(p["l0.w_in"][lay.off_k:lay.off_k + 20], w["l0.mix.left.k"]) and p["l0.w_in"].shape[0] == lay.n_in
    assert torch.equal(p["l0.b_in"][lay.off_v:lay.off_v + 12], w["l0.mix.left.v.b"].float())
    assert torch.equal(p["l0.left.conv_w"].view(2, -1)[1, lay.off_q:lay.off_q + 40], w["l0.mix.left.q.conv"][:, 1].float())
    assert torch.equal(p["l0.w_out"][:, :24], w["l0.mix.left.o"]) and torch.equal(p["l0.w_out"][:, 24:42], w["l0.mix.right.o"])
    assert torch.equal(p["l0.mu"].view(5, -1)[4], w["l0.mix.right.mu.w"].float())
    assert torch.equal(p["l0.w_rkvg"][3], w["l0.mix.right.g"]) and p["l0.w1"].shape == (16, 40)
    assert torch.equal(p["l0.canon_w"].view(4, -1)[0], w["l0.canon1"][:, 0].float())
    assert torch.equal(p["l0.w_ff_in"][24:], w["l0.mlp.up"]) and torch.equal(p["l0.hc2.mix"].view(3, 3), w["l0.hc2.mix"].float())
    assert p["l1.w_in"].shape[0] == 48 and torch.equal(p["l1.w_in"][24:46], w["l1.mix.in"][22:]) and "l1.hc2.in" not in p
    assert torch.equal(p["l1.w_x"][8:18], w["l1.mix.x"][3:]) and float(p["l1.w_x"][3:8].float().abs().max()) == 0.0
    assert torch.equal(p["l1.w_dt"][:, :3], w["l1.mix.dt"]) and p["l1.w_dt"].shape == (22, 8)
    assert torch.equal(p["l2.w_exp_in"][4, 12:], w["l2.mlp.e4.up"]) and torch.equal(p["l2.w_ff_in"][20:40], w["l2.mlp.shared.up"])
    assert p["head"] is p["embed"]


def test_checkpoint_round_trip_with_a_rank_only_the_tensors_know(tmp_path):
    cfg = cfg_small()
    cfg["layers"][0]["mixer"]["right"]["rank"] = 11
    cfg["layers"][2]["mixer"]["rank"] = 5
    spec = models.bibezen_from_config(cfg)
    assert spec.layers[0].wkv.rank == 11 and spec.layers[2].wkv.rank == 5
    w = models.synth_bibezen_weights(spec, seed=2)
    models.save_stack_checkpoint(spec, w, str(tmp_path))
    assert loader.is_stack_model(tmp_path) and "rank" not in (tmp_path / "config.json").read_text().replace("dt_rank", "")
    got, packed = loader.load_model(tmp_path, device="cpu", max_ctx=64, max_slots=2)
    assert got == spec.with_ctx(64, 2)
    want = models.pack_weights(spec, w, device="cpu")
    assert set(packed) == set(want) and all(torch.equal(packed[k], want[k]) for k in want)
    doc = (tmp_path / "config.json").read_text().replace('"streams": 3', '"streams": 2')
    (tmp_path / "config.json").write_text(doc)
    with pytest.raises(loader.LoaderError):      # the tensors are those of three streams
        loader.load_model(tmp_path, device="cpu")


# ------------------------------------------------------------------------------------------ the restatement itself
def small_weights(seed=0):
    cfg = cfg_small()
    return cfg, {k: v.double() for k, v in models.synth_bibezen_weights(models.bibezen_from_config(cfg), seed=seed).items()}


def test_restatement_is_causal_and_depends_on_the_past():
    cfg, w = small_weights()
    g = torch.Generator().manual_seed(3)
    toks = torch.randint(0, 50, (18,), generator=g).tolist()
    a = so.forward(cfg, w, toks)
    other = list(toks)
    other[9] = (toks[9] + 1) % 50
    b = so.forward(cfg, w, other)
    assert torch.equal(a[:9], b[:9]) and all(float((a[t] - b[t]).abs().max()) > 1e-9 for t in range(9, 18))
    assert torch.allclose(so.forward(cfg, w, toks[:11]), a[:11], atol=1e-12)


def test_connections_with_unit_weights_are_a_plain_pre_norm_residual():
    x, y = torch.randn(5, 1, 7), torch.randn(5, 7)
    w = {"p.in": torch.ones(1), "p.out": torch.ones(1), "p.mix": torch.ones(1, 1)}
    assert torch.equal(so.hc_read(x, w, "p."), x[:, 0])
    assert torch.allclose(so.hc_write(x, y, w, "p.", 0.3)[:, 0], x[:, 0] + 0.3 * y)
    x = torch.randn(4, 2, 3)
    w = {"p.mix": torch.tensor([[0.0, 1.0], [0.0, 0.0]]), "p.out": torch.tensor([2.0, 0.0])}   # copy 0 moves to place 1
    y = torch.randn(4, 3)
    out = so.hc_write(x, y, w, "p.", 0.5)
    assert torch.allclose(out[:, 1], x[:, 0]) and torch.allclose(out[:, 0], y)


def test_convolution_last_tap_is_the_current_row():
    u = torch.randn(6, 3)
    assert torch.equal(so.causal_conv(u, torch.tensor([[0.0, 0.0, 1.0]] * 3)), u)
    shifted = so.causal_conv(u, torch.tensor([[0.0, 1.0, 0.0]] * 3))
    assert torch.equal(shifted[1:], u[:-1]) and float(shifted[0].abs().max()) == 0.0


def test_pooled_blocks_and_their_visibility():
    rows = torch.arange(10.0).view(10, 1, 1)
    assert so.pooled_blocks(rows, 3).flatten().tolist() == [1.0, 4.0, 7.0]
    n, size, pool = 30, 7, 4
    tok, blk = so.visible_tokens(n, size), so.visible_blocks(n, n // pool, pool, size)
    for i in range(n):
        for b in range(n // pool):
            assert bool(blk[i, b]) == (not any(bool(tok[i, j]) for j in range(b * pool, b * pool + pool)) and b * pool + pool - 1 < i)


def test_mixed_heads_and_sink():
    cfg, w = small_weights(5)
    m, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    h = torch.randn(12, 40, dtype=torch.float64)
    q, k, v = so.attention_qkv(h, torch.arange(12), m, w, p, 1e-4)
    a = so.attention_weights(q, k, so.pooled_blocks(k, 3), m, w[p + "sink"])
    assert float(a.sum(-1).max()) < 1.0
    b = so.attention_weights(q, k, so.pooled_blocks(k, 3), m, w[p + "sink"], use_sink=False)
    assert torch.allclose(b.sum(-1), torch.ones_like(b.sum(-1)))
    swap = torch.tensor([[0.0, 1, 0, 0], [1, 0, 0, 0], [0, 0, 1, 0], [0, 0, 0, 2]], dtype=torch.float64)
    t = so.talk(a, swap)
    assert torch.equal(t[0], a[1]) and torch.equal(t[1], a[0]) and torch.equal(t[3], 2 * a[3])


def test_time_mixing_bonus_counts_for_the_current_token_only():
    T, H, d = 6, 2, 3
    r, k, v = (torch.randn(T, H, d, dtype=torch.float64) for _ in range(3))
    decay, u = torch.rand(T, H, d, dtype=torch.float64), torch.randn(H, d, dtype=torch.float64)
    out = so.wkv_scan(r, k, v, decay, u)
    for t in range(T):
        want = torch.einsum("hd,hd,hd,hv->hv", r[t], u, k[t], v[t])
        for j in range(t):
            kept = torch.ones(H, d, dtype=torch.float64)
            for i in range(j + 1, t):
                kept = kept * decay[i]
            want = want + torch.einsum("hd,hd,hd,hv->hv", r[t], kept, k[j], v[j])
        assert torch.allclose(out[t], want)


def test_selective_scan_closed_form():
    T, c, n = 5, 3, 2
    x, dt = torch.randn(T, c, dtype=torch.float64), torch.rand(T, c, dtype=torch.float64)
    A, B, C, D = -torch.rand(c, n, dtype=torch.float64), torch.randn(T, n, dtype=torch.float64), torch.randn(T, n, dtype=torch.float64), torch.randn(c, dtype=torch.float64)
    out = so.selective_scan(x, dt, A, B, C, D)
    for t in range(T):
        want = D * x[t]
        for j in range(t + 1):
            kept = torch.exp(dt[j + 1:t + 1].sum(0)[:, None] * A)
            want = want + ((dt[j] * x[j])[:, None] * B[j] * kept * C[t]).sum(1)
        assert torch.allclose(out[t], want)


def test_feed_forwards():
    cfg, w = small_weights(6)
    h = torch.randn(4, 40, dtype=torch.float64)
    m = cfg["layers"][2]["mlp"]
    chosen, weight = so.routing(h, m, w, "l2.mlp.")
    z = h @ w["l2.mlp.router"].T
    assert torch.allclose(weight.sum(-1), torch.ones(4, dtype=torch.float64)) and torch.equal(chosen[:, 0], z.argmax(-1))
    allc = copy.deepcopy(m)
    allc["router"]["top"] = 5
    _, full = so.routing(h, allc, w, "l2.mlp.")
    assert torch.allclose(full, torch.softmax(z, -1).sort(-1, descending=True).values)
    without = {k: v for k, v in m.items() if k != "shared"}
    assert torch.allclose(so.moe_ff(h, m, w, "l2.mlp.") - so.moe_ff(h, without, w, "l2.mlp."), so.gated_ff(h, w, "l2.mlp.shared."))
    big = {"p.gate": torch.full((1, 1), 9.0), "p.up": torch.full((1, 1), -9.0), "p.down": torch.ones(1, 1)}
    lim = torch.tensor(2.0)
    assert torch.allclose(so.dense_ff(torch.ones(1, 1), {"limit": 2.0}, big, "p."), lim * torch.sigmoid(1.702 * lim) * (-lim + 1.0))
