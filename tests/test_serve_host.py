"""Host side of the model-family layer on a machine without a GPU: the registry, config.json / safetensors parsing
and the error paths that end before any CUDA call."""
import json
import math
import os

import pytest
import torch

import nekodra_oracle as O


@pytest.fixture(scope="module")
def S(pkg):
    if not os.path.exists(pkg.lib_path()):
        pytest.fail(f"{pkg.lib_path()} not built: run __graft_entry__.build()")
    return pkg.serve


def test_registry_lists_the_families(S):
    fams = S.lib().b200_model_families().decode().split(",")
    assert "Nekodra" in fams and "Musilorn" in fams and "Tomalix" in fams and "Sakevik" in fams and "Filipel" in fams and "Mazotar" in fams and "llama" in fams


def test_unknown_architecture_and_broken_config(S, tmp_path):
    with pytest.raises(RuntimeError, match="cannot read"):
        S.Model(tmp_path / "nowhere")
    (tmp_path / "config.json").write_text('{"architecture": "Other", "width": 8}')
    with pytest.raises(RuntimeError, match="no family registered"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text('{"architecture": "Nekodra", "width": 8,')
    with pytest.raises(RuntimeError, match="json"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text('{"architecture": "Nekodra", "width": 8}')
    with pytest.raises(RuntimeError, match="required"):
        S.Model(tmp_path)


def test_musilorn_configuration_errors_end_before_any_cuda_call(S, tmp_path):
    (tmp_path / "config.json").write_text('{"architecture": "Musilorn", "width": 8, "vocab": 5, "norm": {"eps": 1e-5}, "layers": []}')
    with pytest.raises(RuntimeError, match="required"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text('{"architecture": "Musilorn", "width": 8, "vocab": 5, "norm": {"eps": 1e-5}, '
                                          '"layers": [{"type": "attention", "mixer": {}, "mlp": null}]}')
    with pytest.raises(RuntimeError, match="residual_mult"):
        S.Model(tmp_path)


def test_tomalix_configuration_errors_end_before_any_cuda_call(S, tmp_path):
    head = '{"architecture": "Tomalix", "width": 8, "vocab": 5, "norm": {"eps": 1e-5}, '
    (tmp_path / "config.json").write_text(head + '"layers": []}')
    with pytest.raises(RuntimeError, match="required"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"layers": [{"type": "retention", "mixer": {}, "mlp": null}]}')
    with pytest.raises(RuntimeError, match="not part of this family"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"layers": [{"type": "attention_2", "mixer": {}, "mlp": {"kind": "glu"}}]}')
    with pytest.raises(RuntimeError, match="feed-forward kind"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"loop": {"start": 0, "stop": 2, "times": 2}, '
                                          '"layers": [{"type": "attention_2", "mixer": {}, "mlp": null}]}')
    with pytest.raises(RuntimeError, match="loop"):
        S.Model(tmp_path)


def test_tomalix_oracle_pieces_agree_with_closed_forms():
    """the plain implementation of the third family: the offset norm, the three frequency rules, the rotation, the block
    mask, the two-map combination, the convolution, the scan against its unrolled sum, the router, the order of layer runs"""
    import tomalix_oracle as T
    g = torch.Generator().manual_seed(2)
    D = torch.float64
    x = torch.randn(4, 6, generator=g, dtype=D)
    assert torch.allclose(T.rms_norm(x, torch.zeros(6, dtype=D), 0.0), x / x.pow(2).mean(-1, keepdim=True).sqrt())
    assert torch.allclose(T.rms_norm(x, torch.full((6,), 0.5, dtype=D), 0.0), 1.5 * T.unit_rms(x, 0.0))
    rot = dict(base=100.0, dims=8)
    plain, amp0 = T.rot_frequencies(rot, "plain")
    lin, amp1 = T.rot_frequencies(dict(rot, scaling=dict(factor=4.0)), "linear")
    assert amp0 == 1.0 and amp1 == 1.0 and torch.allclose(lin, plain / 4) and float(plain[1]) == pytest.approx(100.0 ** (-2 / 8))
    # the ramp: index where `fast` turns fit into `original` positions -> kept; beyond the index of `slow` -> divided by factor
    sc = dict(factor=2.0, original=64, fast=4.0, slow=0.5)
    ramp, amp = T.rot_frequencies(dict(rot, scaling=sc), "ramp")
    idx = lambda turns: 8 * math.log(64 / (2 * math.pi * turns)) / (2 * math.log(100.0))
    lo, hi = max(math.floor(idx(4.0)), 0), min(math.ceil(idx(0.5)), 7)
    assert (lo, hi) == (0, 3) and amp == pytest.approx(0.1 * math.log(2.0) + 1)
    assert ramp[0] == plain[0] and torch.allclose(ramp[3], plain[3] / 2) and torch.allclose(ramp[1], plain[1] * (1 - 1 / 3) + plain[1] / 2 / 3)
    q = torch.randn(5, 2, 8, generator=g, dtype=D)
    r = T.rotate_half(q, dict(base=100.0, dims=4), "plain")
    a = 3 * 100.0 ** (-2 / 4)
    assert torch.equal(r[..., 4:], q[..., 4:]) and torch.equal(r[0], q[0])
    assert torch.allclose(r[3, 1, 1], q[3, 1, 1] * math.cos(a) - q[3, 1, 3] * math.sin(a))
    assert torch.allclose(r[3, 1, 3], q[3, 1, 3] * math.cos(a) + q[3, 1, 1] * math.sin(a))
    m = T.visible(7, 3)
    assert m[5].tolist() == [False, False, False, True, True, True, False] and m[6].tolist() == [False] * 6 + [True]
    assert T.visible(3).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    u, w, b = torch.randn(6, 3, generator=g, dtype=D), torch.randn(3, 4, generator=g, dtype=D), torch.randn(3, generator=g, dtype=D)
    y = T.causal_conv(u, w, b)
    assert torch.allclose(y[0], b + w[:, 3] * u[0]) and torch.allclose(y[5], b + (w.T * u[2:6]).sum(0))
    # the scan of one channel and one state is a weighted sum over the past
    W = {"in": torch.tensor([[1.0], [0.5]], dtype=D), "conv": torch.ones(1, 1, dtype=D),
         "conv.b": torch.zeros(1, dtype=D), "x": torch.tensor([[0.3], [1.0], [2.0]], dtype=D), "dt": torch.ones(1, 1, dtype=D),
         "dt.b": torch.zeros(1, dtype=D), "A_log": torch.zeros(1, 1, dtype=D), "D": torch.tensor([0.25], dtype=D), "o": torch.ones(1, 1, dtype=D)}
    h = torch.randn(4, 1, generator=g, dtype=D)
    got = T.selective_scan(h, dict(inner=1, state=1, dt_rank=1, conv=1), W, "")
    xs, z = T.silu(h[:, 0]), 0.5 * h[:, 0]
    dt = torch.log1p(torch.exp(0.3 * xs))
    want = []
    for t in range(4):
        acc = sum(math.exp(-float(dt[j + 1: t + 1].sum())) * float(dt[j] * xs[j]) * float(xs[j]) for j in range(t + 1))
        want.append((acc * 2.0 * float(xs[t]) + 0.25 * float(xs[t])) * float(T.silu(z[t])))
    assert torch.allclose(got[:, 0], torch.tensor(want, dtype=D))
    # router: the two largest biased logits, weights over those two alone
    Wr = {"router": torch.eye(3, dtype=D), "router.b": torch.tensor([0.0, 0.0, -2.0], dtype=D)}
    for e in range(3):
        Wr["e%d.up" % e], Wr["e%d.down" % e] = torch.full((1, 3), float(e + 1), dtype=D), torch.ones(3, 1, dtype=D)
    hh = torch.tensor([[2.0, 1.0, -1.0]], dtype=D)                     # logits 2, 1, -3: experts 0 and 1
    out = T.routed_ff(hh, dict(router=dict(experts=3, top=2)), Wr, "")
    p = torch.softmax(torch.tensor([2.0, 1.0], dtype=D), 0)
    assert torch.allclose(out[0], (p[0] * 2.0 ** 2 + p[1] * 4.0 ** 2).expand(3))
    cfg = dict(layers=[0, 1, 2, 3], loop=dict(start=1, stop=3, times=2))
    assert T.layer_order(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert T.layer_order(dict(layers=[0, 1])) == [(0, None), (1, None)]


def test_musilorn_oracle_pieces_agree_with_closed_forms():
    """the plain implementation of the second family: rotation pairings, the convolution, the retention walk against its
    unrolled sum, the softmax with one in the denominator, the order in which a repeated span runs"""
    import musilorn_oracle as M
    g = torch.Generator().manual_seed(1)
    x = torch.randn(5, 2, 8, generator=g, dtype=torch.float64)
    rot = dict(base=100.0, dims=4)
    half, inter = M.rotate(x, rot, "half"), M.rotate(x, rot, "interleaved")
    assert torch.equal(half[..., 4:], x[..., 4:]) and torch.equal(inter[0], x[0])          # beyond dims, and position 0
    a = 3 * 100.0 ** (-2 / 4)                                                                # position 3, second frequency
    assert torch.allclose(half[3, 0, 1], x[3, 0, 1] * math.cos(a) - x[3, 0, 3] * math.sin(a))
    assert torch.allclose(inter[3, 0, 3], x[3, 0, 3] * math.cos(a) + x[3, 0, 2] * math.sin(a))
    assert torch.allclose((half ** 2).sum(-1), (x ** 2).sum(-1))                            # a rotation keeps lengths
    f = M.rot_frequencies(dict(base=10000.0, dims=8, scaling=dict(factor=4.0, low=1.0, high=4.0, original=128)))
    plain = M.rot_frequencies(dict(base=10000.0, dims=8))
    assert f[0] == plain[0] and torch.allclose(f[3], plain[3] / 4) and plain[1] / 4 < f[1] < plain[1]
    u, w = torch.randn(6, 3, generator=g, dtype=torch.float64), torch.randn(3, 4, generator=g, dtype=torch.float64)
    y = M.short_conv(u, w)
    assert torch.allclose(y[0], w[:, 3] * u[0]) and torch.allclose(y[5], (w.T * u[2:6]).sum(0))
    q, k, v = (torch.randn(7, n, generator=g, dtype=torch.float64) for n in (4, 4, 5))
    o = M.retention_state_walk(q, k, v, 0.8)
    assert torch.allclose(o[6], sum(0.8 ** (6 - j) * (q[6] @ k[j]) * v[j] for j in range(7)))
    att = M.capped_sink_attention(q, k, v, 0.7, 2.0)
    s = 2.0 * torch.tanh(k[:3] @ q[2] * 0.7 / 2.0)
    assert torch.allclose(att[2], (torch.exp(s) / (1 + torch.exp(s).sum())) @ v[:3])
    cfg = dict(layers=[0, 1, 2, 3], loop=dict(start=1, stop=3, times=2))
    assert M.layer_runs(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]


def test_oracle_pieces_agree_with_torch():
    """the plain implementation itself: its norms and its sink softmax against closed forms"""
    g = torch.Generator().manual_seed(0)
    x, w, b = torch.randn(5, 12, generator=g), torch.randn(12, generator=g), torch.randn(12, generator=g)
    assert torch.allclose(O.layer_norm(x, w, b, 1e-5), torch.nn.functional.layer_norm(x, (12,), w, b, 1e-5), atol=1e-6)
    q, k, v = torch.randn(3, 4, generator=g), torch.randn(6, 4, generator=g), torch.randn(6, 5, generator=g)
    sink = torch.tensor(0.3)
    got = O.sink_attention(q, k, v, 0.5, sink)
    for i in range(3):
        n = 4 + i                                                   # the last three positions of six
        s = torch.cat([(q[i] @ k[:n].T) * 0.5, sink[None]])
        p = torch.softmax(s, 0)[:-1]                                # the sink takes its share and gives nothing back
        assert torch.allclose(got[i], p @ v[:n], atol=1e-6)
    # a very negative sink is plain softmax attention
    plain = O.sink_attention(q, k, v, 0.5, torch.tensor(-1e9))
    assert torch.allclose(plain[2], torch.softmax((q[2] @ k.T) * 0.5, 0) @ v, atol=1e-6)


def test_written_checkpoint_has_the_documented_layout(tmp_path):
    cfg, w = O.random_model(seed=1)
    O.write_model(str(tmp_path), cfg, w)
    raw = (tmp_path / "model.safetensors").read_bytes()
    n = int.from_bytes(raw[:8], "little")
    header = json.loads(raw[8:8 + n])
    assert header["l0.mix.q"]["shape"] == [48, 64] and header["l0.mix.q"]["dtype"] == "BF16"
    assert "l1.mix.dkv" not in header and "l0.mix.dkv" in header    # the second layer reads the first one's rows
    assert json.loads((tmp_path / "config.json").read_text())["layers"][1]["mixer"]["kv_from"] == 0


def test_sakevik_configuration_errors_end_before_any_cuda_call(S, tmp_path):
    head = '{"architecture": "Sakevik", "width": 8, "vocab": 5, "norm": {"eps": 1e-5}, '
    (tmp_path / "config.json").write_text(head + '"layers": []}')
    with pytest.raises(RuntimeError, match="required"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"layers": [{"type": "retention", "mixer": {}, "mlp": null}]}')
    with pytest.raises(RuntimeError, match="not part of this family"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"layers": [{"type": "mingru", "mixer": {"width": 4}, "mlp": {"kind": "moe"}}]}')
    with pytest.raises(RuntimeError, match="feed-forward kind"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"layers": [{"type": "mingru", "mixer": {"width": 4}, "mlp": {"kind": "dense", "ff": 8}}]}')
    with pytest.raises(RuntimeError, match="limit"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"layers": [{"type": "attention", "mixer": {"heads": 3, "kv_heads": 2, "dim": 4, "vdim": 4, '
                                          '"scale": 0.5}, "mlp": null}]}')
    with pytest.raises(RuntimeError, match="multiple of kv_heads"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"layers": [{"type": "latent_attention", "mixer": {"heads": 2, "dim": 4, "vdim": 4, "kv_rank": 6, '
                                          '"rot_dim": 4, "rot": {"base": 100.0, "dims": 2}, "scale": 0.5}, "mlp": null}]}')
    with pytest.raises(RuntimeError, match="rot_dim"):
        S.Model(tmp_path)
    (tmp_path / "config.json").write_text(head + '"embedding": {"scale": 1.0, "bigram": {"buckets": 0, "mul_prev": 1, "mul_cur": 1}}, '
                                          '"layers": [{"type": "mingru", "mixer": {"width": 4}, "mlp": null}]}')
    with pytest.raises(RuntimeError, match="buckets"):
        S.Model(tmp_path)


def test_sakevik_oracle_pieces_agree_with_closed_forms():
    """the plain implementation of the fourth family: the norm, the pair rows, both rotation layouts and their inverse, the
    ramp, the window, the recurrence against its unrolled sum, sigmoid weights that do not sum to one, the clamped unit"""
    import sakevik_oracle as K
    g = torch.Generator().manual_seed(3)
    D = torch.float64
    x = torch.randn(4, 6, generator=g, dtype=D)
    assert torch.allclose(K.rms_norm(x, torch.full((6,), 2.0, dtype=D), 0.0), 2 * x / x.pow(2).mean(-1, keepdim=True).sqrt())
    cfg = dict(embedding=dict(scale=3.0, bigram=dict(buckets=5, mul_prev=7, mul_cur=3)))
    W = dict(embed=torch.randn(9, 2, generator=g, dtype=D), bigram=torch.randn(6, 2, generator=g, dtype=D))
    e = K.embed(cfg, W, [4, 8, 8])
    assert torch.allclose(e[0], 3 * W["embed"][4] + W["bigram"][5]) and torch.allclose(e[1], 3 * W["embed"][8] + W["bigram"][(4 * 7 + 8 * 3) % 5])
    assert torch.allclose(e[2], 3 * W["embed"][8] + W["bigram"][(8 * 7 + 8 * 3) % 5])
    q = torch.randn(5, 2, 6, generator=g, dtype=D)
    ang = K.pair_angles(5, 2, 100.0, 4)
    a = 3 * 100.0 ** (-2 / 4)
    r = K.turn(q, ang, "half")
    assert torch.equal(r[..., 4:], q[..., 4:]) and torch.equal(r[0], q[0])
    assert torch.allclose(r[3, 1, 1], q[3, 1, 1] * math.cos(a) - q[3, 1, 3] * math.sin(a))
    assert torch.allclose(r[3, 1, 3], q[3, 1, 3] * math.cos(a) + q[3, 1, 1] * math.sin(a))
    ri = K.turn(q, ang, "interleaved", 1.5)
    assert torch.allclose(ri[3, 0, 2], 1.5 * (q[3, 0, 2] * math.cos(a) - q[3, 0, 3] * math.sin(a)))
    assert torch.allclose(ri[3, 0, 3], 1.5 * (q[3, 0, 3] * math.cos(a) + q[3, 0, 2] * math.sin(a)))
    assert torch.allclose(K.turn(r, -ang, "half"), q)
    rot = dict(base=100.0, dims=8, scaling=dict(factor=2.0, original=64, fast=4.0, slow=0.5))
    angs, amp = K.ramped_angles(3, rot)
    f = angs[1]
    plain = torch.tensor([100.0 ** (-2 * i / 8) for i in range(4)], dtype=D)
    assert amp == pytest.approx(0.1 * math.log(2.0) + 1) and f[0] == plain[0] and torch.allclose(f[3], plain[3] / 2)
    assert torch.allclose(f[1], plain[1] * (1 - 1 / 3) + plain[1] / 2 / 3)
    m = K.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[1].tolist() == [True, True, False, False, False, False]
    assert K.window_mask(3, 0).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    # one channel: the state is a weighted sum of the candidates, each weight the product of the later keep factors
    Wg = {"z": torch.tensor([[1.0]], dtype=D), "z.b": torch.tensor([0.3], dtype=D), "x": torch.tensor([[2.0]], dtype=D),
          "x.b": torch.tensor([-0.5], dtype=D), "g": torch.tensor([[1.5]], dtype=D), "o": torch.tensor([[1.0]], dtype=D)}
    h = torch.randn(5, 1, generator=g, dtype=D)
    got = K.mingru(h, Wg, "")
    z = torch.sigmoid(h[:, 0] + 0.3)
    u = 2 * h[:, 0] - 0.5
    cand = [float(v + 0.5) if v >= 0 else 1 / (1 + math.exp(-float(v))) for v in u]
    assert any(v >= 0 for v in u) and any(v < 0 for v in u)
    for t in range(5):
        st = sum(float(z[j]) * cand[j] * math.prod(1 - float(z[i]) for i in range(j + 1, t + 1)) for j in range(t + 1))
        assert float(got[t, 0]) == pytest.approx(st * float(K.silu(1.5 * h[t, 0])))
    # two tokens, one head, no rotation on q and k, unit values: the second output sums two sigmoids and need not be below one
    Wa = {"q": torch.zeros(2, 1, dtype=D), "q.b": torch.tensor([1.0, 0.0], dtype=D), "k": torch.zeros(2, 1, dtype=D), "k.b": torch.tensor([1.0, 0.0], dtype=D),
          "v": torch.zeros(2, 1, dtype=D), "v.b": torch.tensor([1.0, 0.0], dtype=D), "q.norm": torch.ones(2, dtype=D), "k.norm": torch.ones(2, dtype=D),
          "pb": torch.tensor([1.0], dtype=D), "g": torch.zeros(1, 1, dtype=D), "o": torch.eye(2, dtype=D), "o.b": torch.zeros(2, dtype=D)}
    mx = dict(heads=1, kv_heads=1, dim=2, vdim=2, scale=0.5, rot=dict(base=100.0, dims=0))
    out = K.sigmoid_attention(torch.zeros(2, 1, dtype=D), mx, Wa, "", 0.0)
    wgt = 1 / (1 + math.exp(-(2.0 * 0.5 + 1.0)))          # normed q and k are (sqrt 2, 0): their product is 2
    assert float(out[0, 0]) == pytest.approx(0.5 * wgt)
    # the value at position 0 is not turned, the one at position 1 by the angle 1; the sum is turned back by 1
    want1 = 0.5 * (wgt * math.cos(-1.0) + wgt)
    assert float(out[1, 0]) == pytest.approx(want1) and 2 * wgt > 1.0
    assert float(K.sigmoid_attention(torch.zeros(2, 1, dtype=D), dict(mx, mask=dict(size=1)), Wa, "", 0.0)[1, 0]) == pytest.approx(0.5 * wgt)
    Wf = {"gate": torch.tensor([[1.0]], dtype=D), "up": torch.tensor([[1.0]], dtype=D), "down": torch.tensor([[1.0]], dtype=D)}
    hv = torch.tensor([[-5.0], [0.5], [5.0]], dtype=D)
    y = K.clamped_glu(hv, dict(limit=2.0), Wf, "")
    assert float(y[2, 0]) == pytest.approx(2.0 / (1 + math.exp(-1.702 * 2.0)) * 3.0)
    assert float(y[1, 0]) == pytest.approx(0.5 / (1 + math.exp(-1.702 * 0.5)) * 1.5)
    assert float(y[0, 0]) == pytest.approx(-5.0 / (1 + math.exp(1.702 * 5.0)) * -1.0)


def test_filipel_configuration_errors_end_before_any_cuda_call(S, tmp_path):
    import json
    lat = dict(type="latent_attention", mixer=dict(heads=2, dim=4, vdim=4, q_rank=5, kv_rank=6, rot_dim=4, scale=0.5, rot=dict(base=100.0, dims=4)), mlp=None)
    par = dict(type="parallel", mixer=dict(left=dict(heads=4, kv_heads=2, dim=4, vdim=4, scale=0.5, rot=dict(base=10.0, dims=4), mask=dict(size=9)),
                                           right=dict(heads=4, vdim=2, state=3, groups=2, conv=4, norm_groups=2)), mlp=None)
    moe = dict(kind="moe", expert=dict(ff=8), router=dict(experts=6, top=2, groups=dict(count=3, keep=2)))

    def refused(layers, text, **top):
        cfg = dict(architecture="Filipel", width=8, vocab=5, norm=dict(eps=1e-5), residual_mult=0.5, layers=layers, **top)
        (tmp_path / "config.json").write_text(json.dumps(cfg))
        with pytest.raises(RuntimeError, match=text):
            S.Model(tmp_path)

    def mixer(base, **kw):
        return dict(base, mixer=dict(base["mixer"], **kw))

    def side(name, **kw):
        return mixer(par, **{name: dict(par["mixer"][name], **kw)})

    def router(**kw):
        return dict(lat, mlp=dict(moe, router=dict(moe["router"], **kw)))
    refused([], "required")
    refused([dict(lat, type="retention")], "not part of this family")
    refused([dict(lat, mixer=None)], "no mixer")
    refused([dict(lat, mlp=dict(kind="glu", ff=8))], "feed-forward kind")
    refused([dict(lat, mlp=dict(kind="dense"))], "mlp.ff")
    refused([mixer(lat, q_rank=0)], "q_rank")
    refused([mixer(lat, rot=dict(base=100.0, dims=2))], "rot_dim")
    refused([mixer(lat, kv_rank=640)], "wider than 640")
    refused([lat, mixer(lat, kv_from=1)], "kv_from")
    refused([par, mixer(lat, kv_from=0)], "kv_from")
    refused([lat, mixer(lat, kv_from=0), mixer(lat, kv_from=1)], "kv_from")
    refused([lat, mixer(lat, kv_from=0, kv_rank=7)], "kv_from: kv_rank")
    refused([lat, mixer(lat, kv_from=0, rot=dict(base=99.0, dims=4))], "kv_from: kv_rank, rot_dim and rotation")
    refused([side("left", heads=3)], "multiple of kv_heads")
    refused([side("left", rot=dict(base=10.0, dims=6))], "at most dim")
    refused([side("left", mask=dict(size=0))], "mask.size")
    refused([side("right", groups=3)], "multiple of groups")
    refused([side("right", norm_groups=3)], "norm_groups")
    refused([side("right", state=300)], "state above 256")
    refused([mixer(par, right=None)], "left and right")
    refused([router(top=7)], "router.top")
    refused([router(groups=dict(count=4, keep=2))], "count must divide")
    refused([router(top=5)], "kept groups must hold")


def test_filipel_random_checkpoint_and_workspaces(S, tmp_path):
    """the random checkpoint names what the loader asks for, and the workspace sizes follow the shape of the step"""
    import json
    par = dict(type="parallel", left=dict(heads=4, kv_heads=2, dim=8, vdim=8, window=9), right=dict(heads=4, vdim=16, state=8, groups=1, conv=4, norm_groups=1))
    lat = dict(type="latent_attention", heads=2, dim=8, rot_dim=4, vdim=8, q_rank=12, kv_rank=16)
    cfg, w = S.random_filipel(32, 50, [dict(lat, ff=24), dict(par, ff=(8, 4, 2, 2, 1)), dict(lat, kv_from=0, ff=None)])
    S.write_checkpoint(tmp_path, cfg, w)
    raw = (tmp_path / "model.safetensors").read_bytes()
    header = json.loads(raw[8:8 + int.from_bytes(raw[:8], "little")])
    assert header["l1.mix.right.in"]["shape"] == [64 + 64 + 16 + 4, 32] and header["l1.mix.left.talk"]["shape"] == [4, 4]
    assert "l0.mix.dkv" in header and "l2.mix.dkv" not in header and header["l0.mlp.act"]["shape"] == [4]
    assert header["l1.mlp.e3.down"]["shape"] == [32, 8] and "l2.mlp.up" not in header
    L = S.lib()
    assert L.b200_mixed_attention_workspace_bytes(1, 4, 9, 100) == 0                     # a single token needs none
    few, many = L.b200_mixed_attention_workspace_bytes(100, 4, 9, 5000), L.b200_mixed_attention_workspace_bytes(100, 4, 0, 5000)
    assert few == 128 * (4 * 192 * 6 + 4 * 8 + 8) and many > 20 * few                     # 9 + 126 columns in whole tiles; no window: all
    assert L.b200_mixed_attention_workspace_bytes(1 << 20, 16, 1024, 1 << 20) <= 256 << 20   # long prompts go block by block
    assert L.b200_ssd_scan_workspace_bytes(127, 1, 4, 1, 16, 8) == 0 and L.b200_ssd_scan_workspace_bytes(128, 1, 4, 1, 16, 8) >= 4 * 4 * 16 * 8 * 4


def test_filipel_oracle_pieces_agree_with_closed_forms():
    """the plain implementation of the fifth family: both norms, the window, the mix, the recurrence against its unrolled sum, the
    convolution, the normed powers, the router's groups"""
    import filipel_oracle as K
    g = torch.Generator().manual_seed(3)
    D = torch.float64
    x = torch.randn(4, 6, generator=g, dtype=D)
    n = K.layer_norm(x, torch.full((6,), 2.0, dtype=D), 0.0)
    assert torch.allclose(n.mean(-1), torch.zeros(4, dtype=D), atol=1e-12) and torch.allclose(n.pow(2).mean(-1), torch.full((4,), 4.0, dtype=D))
    assert torch.allclose(K.rms_norm(x, torch.ones(6, dtype=D), 0.0).pow(2).mean(-1), torch.ones(4, dtype=D))
    m = K.visible(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[1].tolist() == [True, True, False, False, False, False]
    assert K.visible(3, 0).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    q = torch.randn(5, 2, 6, generator=g, dtype=D)
    r = K.turn_half(q, dict(base=100.0, dims=4))
    a = 3 * 100.0 ** (-2 / 4)
    assert torch.equal(r[..., 4:], q[..., 4:]) and torch.equal(r[0], q[0])
    assert torch.allclose(r[3, 1, 1], q[3, 1, 1] * math.cos(a) - q[3, 1, 3] * math.sin(a))
    assert torch.allclose(r[3, 1, 3], q[3, 1, 3] * math.cos(a) + q[3, 1, 1] * math.sin(a))
    # two heads, two positions, zero queries: every weight of position 1 is a half; the mix acts on the heads
    talk = torch.tensor([[1.0, 2.0], [0.0, -1.0]], dtype=D)
    v = torch.tensor([[[1.0]], [[3.0]]], dtype=D)
    o = K.mixed_attention(torch.zeros(2, 2, 1, dtype=D), torch.zeros(2, 1, 1, dtype=D), v, 1.0, torch.ones(2, dtype=D), talk, 0)
    assert torch.allclose(o[:, :, 0], torch.tensor([[3.0, -1.0], [6.0, -2.0]], dtype=D))
    o = K.mixed_attention(torch.zeros(2, 2, 1, dtype=D), torch.zeros(2, 1, 1, dtype=D), v, 1.0, torch.ones(2, dtype=D), talk, 1)
    assert torch.allclose(o[1, :, 0], torch.tensor([9.0, -3.0], dtype=D))
    # temperature: ln 3 times the score difference of one
    o = K.mixed_attention(torch.ones(2, 1, 1, dtype=D), torch.tensor([[[0.0]], [[1.0]]], dtype=D), v, 1.0, torch.tensor([math.log(3.0)], dtype=D),
                          torch.ones(1, 1, dtype=D), 0)
    assert float(o[1, 0, 0]) == pytest.approx(0.25 * 1 + 0.75 * 3)
    # one head, one state, one column: the output is a sum over older inputs, each decayed by every later step
    B, Cc, xs, dt = (torch.rand(5, generator=g, dtype=D) for _ in range(4))
    y = K.ssd(xs.view(5, 1, 1), B.view(5, 1, 1), Cc.view(5, 1, 1), dt.view(5, 1), torch.tensor([0.4], dtype=D), torch.tensor([0.7], dtype=D))
    for t in range(5):
        want = 0.7 * xs[t] + sum(Cc[t] * B[j] * dt[j] * xs[j] * math.exp(-math.exp(0.4) * float(dt[j + 1:t + 1].sum())) for j in range(t + 1))
        assert float(y[t, 0, 0]) == pytest.approx(float(want))
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=D)
    c = K.causal_conv_silu(u, torch.tensor([[10.0, 1.0]], dtype=D), torch.tensor([0.5], dtype=D))
    assert torch.allclose(c[:, 0], K.silu(torch.tensor([1.5, 12.5, 24.5], dtype=D)))
    z = torch.tensor([[1.0, -2.0]], dtype=D)
    p = K.poly_norm(z, (1.0, 0.5, 2.0, 0.25), 0.0)
    want = [s / math.sqrt(2.5) + 0.5 * s * s / math.sqrt(8.5) + 2 * s ** 3 / math.sqrt(32.5) + 0.25 for s in (1.0, -2.0)]
    assert p[0].tolist() == pytest.approx(want)
    # the second largest logit lies in a group that is not kept
    logits = torch.log(torch.tensor([[8.0, 1.0, 7.0, 0.5, 6.0, 5.0]], dtype=D))
    chosen, w = K.route(logits, dict(count=3, keep=1), 2)
    assert chosen.tolist() == [[0, 1]] and w[0].tolist() == pytest.approx([8 / 9, 1 / 9])
    chosen, w = K.route(logits, None, 2)
    assert chosen.tolist() == [[0, 2]] and w[0].tolist() == pytest.approx([8 / 15, 7 / 15])
    gn = K.gated_group_norm(torch.ones(1, 4, dtype=D), torch.tensor([[1.0, 1.0, 5.0, 5.0]], dtype=D), torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=D), 2, 0.0)
    assert torch.allclose(gn, torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=D))


def test_mazotar_configuration_errors_end_before_any_cuda_call(S, tmp_path):
    import json
    att = dict(type="attention", mixer=dict(heads=4, kv_heads=2, dim=4, vdim=6, scale=0.5, bias_max=30, q_temp=dict(coef=0.1, every=8)), mlp=None)
    mem = dict(type="mlstm", mixer=dict(heads=2, dim=4, vdim=6, gate_cap=9.0), mlp=None)
    moe = dict(kind="moe", expert=dict(ff=8), router=dict(experts=6, top=2), shared=dict(ff=4))

    def refused(layers, text, **top):
        cfg = dict(dict(architecture="Mazotar", width=8, vocab=5, streams=2, norm=dict(eps=1e-5), embedding=dict(scale=1.0), layers=layers), **top)
        (tmp_path / "config.json").write_text(json.dumps(cfg))
        with pytest.raises(RuntimeError, match=text):
            S.Model(tmp_path)

    def mixer(base, **kw):
        return dict(base, mixer=dict(base["mixer"], **kw))
    refused([], "required")
    refused([att], "streams must be positive", streams=0)
    refused([att], "16 streams", streams=17)
    refused([dict(att, type="retention")], "not part of this family")
    refused([dict(att, mixer=None)], "no mixer")
    refused([dict(att, mlp=dict(kind="glu", ff=8))], "feed-forward kind")
    refused([dict(mem, mlp=dict(kind="dense"))], "mlp.ff")
    refused([dict(mem, mlp=dict(moe, shared=dict()))], "mlp.shared.ff")
    refused([dict(mem, mlp=dict(moe, router=dict(experts=6, top=7)))], "router.top")
    refused([dict(mem, mlp=dict(moe, router=dict(experts=60, top=17)))], "16 experts")
    refused([mixer(att, bias_max=0)], "bias_max")
    refused([mixer(att, heads=3)], "multiple of kv_heads")
    refused([mixer(att, vdim=257)], "above 256")
    refused([mixer(att, q_temp=dict(coef=0.1, every=0))], "q_temp.every")
    refused([att, mixer(att, kv_from=1)], "kv_from")
    refused([mem, mixer(att, kv_from=0)], "kv_from")
    refused([att, mixer(att, kv_from=0), mixer(att, kv_from=1)], "kv_from")
    refused([att, mixer(att, kv_from=0, vdim=5)], "kv_from: kv_heads, dim and vdim")
    refused([mixer(mem, gate_cap=0.0)], "gate_cap")
    refused([mixer(mem, dim=513)], "above 512")


def test_mazotar_random_checkpoint_and_workspaces(S, tmp_path):
    """the random checkpoint names what the loader asks for, and the workspace sizes follow the shape of the step"""
    import json
    att = dict(type="attention", heads=4, kv_heads=2, dim=8, vdim=8, buckets=6, bias_max=40)
    cfg, w = S.random_mazotar(32, 50, [dict(type="mlstm", heads=2, dim=4, vdim=6, ff=24), dict(att, ff=(8, 4, 2, 16)), dict(att, kv_from=1, ff=None)], streams=3)
    S.write_checkpoint(tmp_path, cfg, w)
    raw = (tmp_path / "model.safetensors").read_bytes()
    header = json.loads(raw[8:8 + int.from_bytes(raw[:8], "little")])
    assert header["l0.mix.i.b"]["shape"] == [2] and header["l0.mix.norm"]["shape"] == [12] and header["l1.mix.rel"]["shape"] == [6, 4]
    assert "l1.mix.k.norm" in header and "l2.mix.k" not in header and "l2.mix.k.norm" not in header and "l2.hc2.in" not in header
    assert header["l1.hc2.mix"]["shape"] == [3, 3] and header["l1.mlp.shared.sg"]["shape"] == [1, 32] and header["l1.mlp.e3.down"]["shape"] == [32, 8]
    L = S.lib()
    assert L.b200_mlstm_norm_floats(8, 32) == 12 and L.b200_mlstm_norm_floats(9, 130) == 3 * 16     # n, padding, the maximum; a copy per 64 columns
    assert L.b200_mlstm_workspace_bytes(127, 1, 4, 16, 8) == 0 and L.b200_mlstm_workspace_bytes(1000, 1, 4, 300, 8) == 0
    assert L.b200_mlstm_workspace_bytes(128, 2, 4, 16, 8) >= 5 * 4 * (16 * 8 + 16 + 64 * 64 + 64) * 4


def test_mazotar_oracle_pieces_agree_with_closed_forms():
    """the plain implementation of the sixth family: sinusoids, buckets, the sink, the temperature, the memory against its unrolled
    sum, the streams"""
    import mazotar_oracle as K
    g = torch.Generator().manual_seed(3)
    D = torch.float64
    s = K.sinusoids(4, 5)
    assert s[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0] and float(s[3, 2]) == pytest.approx(math.sin(3 * 10000 ** (-2 / 5)))
    assert float(s[3, 3]) == pytest.approx(math.cos(3 * 10000 ** (-2 / 5)))
    assert [K.bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 9999)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    b = K.distance_bias(6, torch.tensor([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0], [4.0, 40.0]], dtype=D), 8)
    assert b[0, 5].tolist() == [4.0, 4.0, 3.0, 3.0, 2.0, 1.0] and b[1, 2].tolist() == [30.0, 20.0, 10.0, 0.0, 0.0, 0.0]
    assert K.temperature(4, 0.5, 2).tolist() == pytest.approx([1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)])
    p = K.sink_softmax(torch.log(torch.tensor([[[1.0, 3.0]]], dtype=D)), torch.log(torch.tensor([4.0], dtype=D)))
    assert p[0, 0].tolist() == pytest.approx([1 / 8, 3 / 8])
    # zero queries: the weights are exp(bias) over their sum and the sink
    v = torch.tensor([[[1.0]], [[5.0]]], dtype=D)
    o = K.attend(torch.zeros(2, 1, 1, dtype=D), torch.ones(2, 1, 1, dtype=D), v, 1.0, torch.log(torch.tensor([[[2.0, 1.0], [6.0, 2.0]]], dtype=D)), torch.zeros(1, dtype=D))
    assert o[:, 0, 0].tolist() == pytest.approx([2 / 3, (6 * 1 + 2 * 5) / 9])
    # one head: the memory is a sum over older tokens; with the maximum taken out the floor of the denominator is 1
    q, k, x, i = (torch.rand(5, generator=g, dtype=D) for _ in range(4))
    f = -torch.rand(5, generator=g, dtype=D)
    i = i * 3 - 1
    y = K.mlstm_memory(q.view(5, 1, 1), k.view(5, 1, 1), x.view(5, 1, 1), i.view(5, 1), f.view(5, 1))
    m = 0.0
    for t in range(5):
        m = max(float(f[t]) + m, float(i[t]))
        wts = [math.exp(float(i[j] + f[j + 1:t + 1].sum())) for j in range(t + 1)]
        num, den = sum(w_ * k[j] * x[j] for j, w_ in enumerate(wts)) * q[t], abs(sum(w_ * k[j] for j, w_ in enumerate(wts)) * q[t])
        assert float(y[t, 0, 0]) == pytest.approx(float(num / (max(den, 1.0) + 1e-6 * math.exp(m))))
    assert float(K.capped(torch.tensor(100.0, dtype=D), 7.0)) == pytest.approx(7.0)
    chosen, w = K.route(torch.tensor([[0.0, math.log(3.0), -1.0]], dtype=D), 2)
    assert chosen.tolist() == [[1, 0]] and w[0].tolist() == pytest.approx([0.75, 0.5])
    W = {"in": torch.tensor([1.0, 2.0], dtype=D), "mix": torch.tensor([[1.0, 3.0], [0.0, 1.0]], dtype=D), "out": torch.tensor([1.0, -1.0], dtype=D)}
    n = K.hyper(torch.tensor([[[3.0]], [[-1.0]]], dtype=D), W, "", torch.tensor([2.0], dtype=D), 0.0, lambda h: h * 5)
    assert n[:, 0, 0].tolist() == [3.0 + 10.0, 3.0 * 3 - 1 - 10.0]     # u = 1, normed and weighted to 2, y = 10


def test_every_registered_family_has_a_program_of_its_own(S):
    """bin/trace_run compiles one family's objects: the build has to know every family that the registry knows (llama is served by the
    whole library)"""
    import pathlib
    import subprocess
    pkg_dir = pathlib.Path(__file__).resolve().parent.parent / "llm-inference_b200"
    known = subprocess.run(["make", "-s", "--no-print-directory", "-C", str(pkg_dir), "serve_families"], capture_output=True, text=True, check=True).stdout.split()
    assert set(known) == set(S.lib().b200_model_families().decode().split(",")) - {"llama"}
