"""The Filipel family through the library's own entry points (registry -> step function -> paged cache and slot state ->
scheduler) against the plain implementation in filipel_oracle.py, on small random models of several shapes: whole prompts
with every layer, prefill against token-by-token decoding, prompt portions down to two tokens, unequal batches against each
request alone, pages, slots, states and convolution inputs that are freed and used again, window and page borders in prompts
and in decoding, the first tokens of a sequence, long decoding, sizes that are 1 or equal to each other, and greedy
generation through the continuous-batching scheduler."""
import copy

import numpy as np
import pytest
import torch

import filipel_oracle as O

pytestmark = pytest.mark.gpu


def lat(H, d, dr, dv, q_rank, R, **kw):
    return dict(type="latent_attention", heads=H, dim=d, rot_dim=dr, vdim=dv, q_rank=q_rank, kv_rank=R, **kw)


def par(left, right, **kw):
    return dict(type="parallel", left=dict(zip(("heads", "kv_heads", "dim", "vdim", "window"), left[:5]), **left[5]),
                right=dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right)), **kw)


SHAPES = {
    # every branch: both mixers with a dense, a routed and no feed-forward; a layer on another layer's rows; windows of 37 and 21
    # beside pages of 64; experts in groups
    "mix": dict(width=48, vocab=61, mult=0.6, layers=[
        lat(4, 8, 4, 12, 20, 24, base=50.0, ff=40),
        par((4, 2, 16, 8, 37, dict(rot_dims=8, base=100.0)), (4, 6, 10, 2, 4, 2), ff=(16, 10, 3, 5, 3)),
        lat(6, 4, 4, 6, 12, 24, base=50.0, scale=0.4, kv_from=0, ff=None),
        par((2, 1, 8, 12, 21, dict(base=30.0)), (2, 12, 7, 1, 3, 1), ff=24),
        lat(4, 8, 6, 8, 9, 16, base=200.0, ff=(12, 6, 2, 3, 1))]),
    # sizes that are 1 or equal; one tap, one state, one head; a window of one position and none at all; no rotation; experts
    # without groups and one expert in all; a parallel layer first; a multiplier of one
    "odd": dict(width=40, vocab=33, mult=1.0, eps=1e-3, layers=[
        par((1, 1, 4, 2, 1, dict(rot_dims=0)), (1, 1, 1, 1, 1, 1), ff=(8, 1, 1, 1, 1)),
        lat(1, 1, 2, 1, 1, 3, ff=None),
        par((6, 1, 6, 5, None, dict(rot_dims=4)), (3, 5, 9, 3, 2, 3), ff=None),
        lat(3, 10, 6, 6, 40, 40, scale=0.5, ff=(8, 5, 3, None, None)),
        lat(5, 6, 6, 3, 7, 40, scale=0.3, base=10000.0, kv_from=3, ff=1)]),
    # nothing a multiple of 8
    "plain": dict(width=36, vocab=41, mult=0.25, layers=[
        par((5, 5, 10, 6, 33, dict(rot_dims=10)), (6, 3, 5, 2, 5, 9), ff=(20, 9, 2, 3, 2)),
        lat(5, 6, 6, 9, 13, 11, ff=20),
        par((3, 3, 10, 7, 5, dict(rot_dims=6, base=7.0)), (2, 9, 17, 2, 2, 1), ff=(12, 4, 4, 2, 2))]),
    # heads as wide as the tensor-core tiles take them, windows long enough for clusters, states that fill the chunk tiles
    "wide": dict(width=64, vocab=50, mult=0.5, layers=[
        par((8, 2, 64, 64, 100, dict()), (4, 64, 64, 1, 4, 4), ff=128),
        lat(8, 32, 32, 32, 48, 96, ff=(64, 8, 2, 4, 2)),
        par((16, 16, 32, 48, 300, dict(rot_dims=16, base=500.0)), (2, 72, 128, 2, 4, 1), ff=(32, 16, 4, 4, 2)),
        lat(4, 64, 32, 64, 32, 96, kv_from=1, ff=64)]),
}
RTOL = {"f32": 3e-4, "bf16": 6e-2}


@pytest.fixture(scope="module")
def S(pkg):
    if not torch.cuda.is_available():
        pytest.fail("no CUDA device: the library has no CPU path")
    return pkg.serve


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, sh) in enumerate(SHAPES.items()):
        cfg, w = O.random_model(seed=90 + i, **sh)
        folder = tmp_path_factory.mktemp(name)
        O.write_model(str(folder), cfg, w)
        out[name] = (str(folder), O.Oracle(cfg, w), cfg)
    return out


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(got, want):
    """per row: rms of the difference with its mean taken off, over the rms of the wanted row"""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return (np.sqrt((d ** 2).mean(-1)) / np.sqrt((want ** 2).mean(-1))).reshape(-1)


def err(got, want):
    return float(row_errors(got, want).max())


def check(got, want, kind, what=""):
    """fp32: every row within the tolerance. bfloat16: the norms on both mixer outputs and a router's close calls turn the
    rounding of a small output into a change of its direction; so nine rows in ten have to be within the tolerance and the
    median well inside it."""
    e = row_errors(got, want)
    assert np.all(np.isfinite(e)), what
    if kind == "f32":
        assert e.max() < RTOL[kind], (what, float(e.max()), int(e.argmax()))
    else:
        assert np.quantile(e, 0.9) < RTOL[kind] and np.median(e) < RTOL[kind] / 2, (what, float(np.quantile(e, 0.9)), float(np.median(e)))


def open_model(S, folder, kind, max_tokens=1024, slots=4):
    return S.Model(folder, dtype=S.BF16 if kind == "bf16" else S.F32, max_tokens=max_tokens, max_slots=slots)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_whole_prompt_and_every_layer(S, models, name, kind):
    folder, oracle, cfg = models[name]
    m = open_model(S, folder, kind)
    assert m.family == "Filipel" and m.vocab == cfg["vocab"] and m.n_layers == len(cfg["layers"])
    toks = tokens(150, cfg["vocab"], 1)
    m.capture_layers(True)
    got = m.step([(0, toks, list(range(150)))])
    want, trail = oracle.forward(toks, return_layers=True)
    layers = m.captured_layers(150)
    for i in range(len(cfg["layers"])):
        check(layers[i], trail[i].numpy(), kind, f"residual after layer {i}")
    check(got, want.numpy(), kind)
    assert m.step_launches > 0
    m.close()


def test_every_mechanism_reaches_the_logits(models):
    """sensitivity of the comparison itself: with a window one position off, the mix, the temperatures, the gates, the rotation,
    the shared rows, the groups, the convolution, the decays, the direct term, the norms or a constant changed, the oracle's
    logits move by far more than the tolerance the library is held to"""
    _, oracle, cfg = models["mix"]
    toks = tokens(90, cfg["vocab"], 2)
    base = oracle.forward(toks).numpy()

    def moved(change_cfg=None, change_w=None):
        c, w = copy.deepcopy(cfg), dict(oracle.w)
        if change_cfg:
            change_cfg(c)
        if change_w:
            change_w(w)
        return err(O.Oracle(c, w).forward(toks).numpy(), base)

    def window(c): c["layers"][1]["mixer"]["left"]["mask"]["size"] = 36
    def window_wide(c): c["layers"][3]["mixer"]["left"]["mask"]["size"] = 22
    def base_left(c): c["layers"][1]["mixer"]["left"]["rot"]["base"] = 90.0
    def base_latent(c): c["layers"][0]["mixer"]["rot"]["base"] = 45.0
    def keep(c): c["layers"][1]["mlp"]["router"]["groups"]["keep"] = 2
    def one_group(c): del c["layers"][4]["mlp"]["router"]["groups"]
    def mult(c): c["residual_mult"] = 0.59
    def eps(c): c["norm"]["eps"] = 1e-2
    def parts(c): c["layers"][1]["mixer"]["right"]["norm_groups"] = 4
    def scale(c): c["layers"][2]["mixer"]["scale"] = 0.41
    for change in (window, window_wide, base_left, base_latent, keep, one_group, mult, eps, parts, scale):
        assert moved(change_cfg=change) > 10 * RTOL["f32"], change.__name__

    def changed(name, f):
        def change(w): w[name] = f(w[name])
        change.__name__ = name
        return change
    for change in (changed("l1.mix.left.talk", lambda t: torch.eye(4, dtype=O.DT)), changed("l1.mix.left.talk", lambda t: t.T.contiguous()),
                   changed("l1.mix.left.temp", torch.ones_like), changed("l1.mix.left.g", torch.zeros_like), changed("l0.mix.g", torch.zeros_like),
                   changed("l1.mix.left.out", torch.ones_like), changed("l1.mix.right.out", torch.ones_like), changed("l1.mix.right.norm", torch.ones_like),
                   changed("l1.mix.right.conv.b", torch.zeros_like), changed("l1.mix.right.conv", lambda t: t.flip(1)),
                   changed("l1.mix.right.dt_bias", torch.zeros_like), changed("l1.mix.right.A_log", torch.zeros_like),
                   changed("l1.mix.right.D", torch.zeros_like), changed("l0.mix.dq.norm", torch.ones_like), changed("l0.mix.dkv.norm", torch.ones_like),
                   changed("l0.mlp.act", lambda t: t * torch.tensor([1.0, 1.0, 1.0, 0.0], dtype=O.DT)),
                   changed("l0.mlp.act", lambda t: t[[0, 2, 1, 3]])):
        assert moved(change_w=change) > 10 * RTOL["f32"], change.__name__


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mix", "odd", "plain"])
def test_prefill_against_token_by_token_decoding(S, models, name, kind):
    """70 tokens in one step, then 80 one by one across the page border at 128 and past every window; and a second sequence
    decoded from its very first token (its states and convolution inputs start at zero)"""
    folder, oracle, cfg = models[name]
    toks = tokens(150, cfg["vocab"], 3)
    want = oracle.forward(toks).numpy()
    m = open_model(S, folder, kind)
    got = [m.step([(0, toks[:70], list(range(70)))])]
    for t in range(70, 150):
        got.append(m.step([(0, [toks[t]], [0])]))
    check(np.concatenate(got), want, kind, "prompt then single tokens")
    got = [m.step([(1, [toks[t]], [0])]) for t in range(40)]
    check(np.concatenate(got), want[:40], kind, "single tokens from the first position")
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mix", "odd", "wide"])
def test_portions_of_many_sizes(S, models, name, kind):
    """the same prompt cut into portions of 1 .. 64 tokens (ending inside windows, convolution taps and pages)"""
    folder, oracle, cfg = models[name]
    toks = tokens(200, cfg["vocab"], 4)
    want = oracle.forward(toks).numpy()
    m = open_model(S, folder, kind)
    cuts, at = [2, 3, 2, 37, 5, 2, 64, 1, 1, 2, 29, 31, 2, 19], 0
    got = []
    for c in cuts:
        got.append(m.step([(0, toks[at: at + c], list(range(c)))]))
        at += c
    assert at == 200
    check(np.concatenate(got), want, kind)
    m.close()


@pytest.mark.parametrize("name", ["mix", "plain", "wide"])
def test_a_position_does_not_depend_on_the_cut_or_the_batch(S, models, name):
    """fp32: three unequal requests batched together (portions beside single tokens) against each alone in one step"""
    folder, oracle, cfg = models[name]
    V = cfg["vocab"]
    reqs = [tokens(90, V, 10), tokens(33, V, 11), tokens(140, V, 12)]
    m = open_model(S, folder, "f32")
    alone = []
    for r in reqs:
        alone.append(m.step([(3, r, list(range(len(r))))]))
        m.release(3)
    got = [[], [], []]
    plan = [[(0, 40), (1, 3), (2, 64)], [(0, 1), (1, 2), (2, 2)], [(0, 1), (2, 70)], [(0, 48), (1, 28), (2, 1)], [(2, 1)], [(2, 1)], [(2, 1)]]
    at = [0, 0, 0]
    for stp in plan:
        entries = [(i, reqs[i][at[i]: at[i] + c], list(range(c))) for i, c in stp]
        out = m.step(entries)
        o = 0
        for i, c in stp:
            got[i].append(out[o: o + c])
            o += c
            at[i] += c
    for i in range(3):
        assert at[i] == len(reqs[i])
        assert err(np.concatenate(got[i]), alone[i]) < 2e-5, i
        assert err(alone[i], oracle.forward(reqs[i]).numpy()) < RTOL["f32"]
    m.close()


@pytest.mark.parametrize("name", ["mix", "wide"])
def test_a_batch_of_portions_and_single_tokens_in_bfloat16(S, models, name):
    """the tile and chunk kernels on entries of 130, 2, 1 and 60 tokens in one step (chunk form for all of them), then single
    tokens of all four"""
    folder, oracle, cfg = models[name]
    V = cfg["vocab"]
    first, then = [130, 2, 1, 60], [1, 1, 1, 1]
    reqs = [tokens(n + 3, V, 60 + n) for n in first]
    m = open_model(S, folder, "bf16")
    m.step([(2, reqs[2][:1], []), (1, reqs[1][:1], [])])     # two of them have a token behind them already
    at = [0, 1, 1, 0]
    got = [[], [], [], []]
    for counts in (first, then, then):
        entries = [(i, reqs[i][at[i]: at[i] + min(c, len(reqs[i]) - at[i])], None) for i, c in enumerate(counts)]
        entries = [(i, t, list(range(len(t)))) for i, t, _ in entries if t]
        out, o = m.step(entries), 0
        for i, t, _ in entries:
            got[i].append(out[o: o + len(t)])
            o += len(t)
            at[i] += len(t)
    for i in range(4):
        check(np.concatenate(got[i]), oracle.forward(reqs[i][:at[i]]).numpy()[-sum(len(x) for x in got[i]):], "bf16", f"request {i}")
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_pages_slots_and_states_used_again(S, models, kind):
    """a pool of three pages and two slots: requests follow one another through the same pages, recurrent states and convolution
    inputs, which still hold what the previous owner left; an oversized step is refused without side effects"""
    folder, oracle, cfg = models["mix"]
    V = cfg["vocab"]
    m = open_model(S, folder, kind, max_tokens=192, slots=2)
    assert m.pages_total == 3
    for rnd in range(3):
        a, b = tokens(100, V, 20 + rnd), tokens(50, V, 30 + rnd)
        ga = [m.step([(0, a[:60], list(range(60)))])]
        gb = [m.step([(1, b[:10], list(range(10)))])]
        out = m.step([(0, a[60:], list(range(40))), (1, b[10:], list(range(40)))])
        ga.append(out[:40]); gb.append(out[40:])
        check(np.concatenate(ga), oracle.forward(a).numpy(), kind, f"turn {rnd}, first request")
        check(np.concatenate(gb), oracle.forward(b).numpy(), kind, f"turn {rnd}, second request")
        free = m.pages_free
        with pytest.raises(RuntimeError):
            m.step([(1, tokens(80, V, 1), [0])])          # 50 + 80 tokens need a third page for slot 1: none left
        assert m.pages_free == free and m.slot_length(1) == 50
        m.release(0)
        m.release(1)
        assert m.pages_free == 3
    m.close()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mix", "wide"])
def test_long_decoding(S, models, name, kind):
    folder, oracle, cfg = models[name]
    n = 330 if name == "mix" else 420
    toks = tokens(n, cfg["vocab"], 5)
    want = oracle.forward(toks).numpy()
    m = open_model(S, folder, kind)
    got = [m.step([(0, toks[:10], list(range(10)))])]
    for t in range(10, n):     # the same single-token shape again and again: graph replay, windows that slide, page borders
        got.append(m.step([(0, [toks[t]], [0])]))
    check(np.concatenate(got), want, kind)
    m.close()


def test_long_prompt_in_one_step_and_in_portions(S, models):
    """700 tokens: the recurrence's chunk form, attention tiles over many key tiles, windows far from the sequence's start,
    against the same prompt in odd portions"""
    folder, oracle, cfg = models["wide"]
    toks = tokens(700, cfg["vocab"], 6)
    want = oracle.forward(toks).numpy()
    for kind in ("f32", "bf16"):
        m = open_model(S, folder, kind, max_tokens=2048)
        whole = m.step([(0, toks, list(range(700)))])
        check(whole, want, kind, "one step")
        got, at = [], 0
        for c in [301, 257, 2, 140]:
            got.append(m.step([(1, toks[at: at + c], list(range(c)))]))
            at += c
        check(np.concatenate(got), want, kind, "portions")
        if kind == "f32":
            assert err(np.concatenate(got), whole) < 2e-5
        m.close()


def test_experts_of_a_long_prompt_as_dense_products(S, tmp_path):
    """a bfloat16 step of more than a thousand tokens with experts wide enough for the dense products per expert"""
    cfg, w = O.random_model(seed=3, width=64, vocab=40, layers=[lat(2, 16, 8, 16, 24, 32, ff=(128, 6, 2, 3, 2)),
                                                                par((4, 2, 16, 16, 50, dict()), (2, 16, 16, 1, 4, 1), ff=(128, 4, 2, 2, 1))])
    O.write_model(str(tmp_path), cfg, w)
    toks = tokens(1100, 40, 7)
    m = open_model(S, str(tmp_path), "bf16", max_tokens=2048)
    got = m.step([(0, toks, list(range(1100)))])
    many = m.step_launches
    check(got, O.forward(cfg, w, toks).numpy(), "bf16")
    m.release(0)
    parts = [m.step([(0, toks[:900], list(range(900)))]), m.step([(0, toks[900:], list(range(200)))])]     # the grouped kernel
    assert m.step_launches < many
    check(np.concatenate(parts), got, "bf16")
    m.close()


def test_a_key_at_the_window_edge_decides_the_logits(S, tmp_path):
    """one parallel layer in which every query points along one direction and only the token `mark` has its key there: its
    value takes the whole softmax of every head while it is inside the window, and is gone one position later. The library has
    to follow the oracle on both sides, for prompt rows and for single tokens."""
    cfg, w = O.random_model(seed=5, width=32, vocab=30, layers=[par((2, 1, 8, 8, 20, dict(rot_dims=0, scale=4.0)), (1, 4, 2, 1, 2, 1), ff=None)])
    mark = 7
    h = O.layer_norm(w["embed"], w["l0.norm1"], 1e-5)
    rest = h[[i for i in range(30) if i != mark]]
    # a direction that the marked token's normed row has and the others' have little of (least squares)
    a = torch.linalg.lstsq(torch.cat([rest, h[mark:mark + 1] * 8]), torch.cat([torch.zeros(29, 1, dtype=O.DT), torch.full((1, 1), 8.0, dtype=O.DT)])).solution[:, 0]
    b = torch.linalg.lstsq(h, torch.ones(30, 1, dtype=O.DT)).solution[:, 0]          # about one for every token
    lp = "l0.mix.left."
    w[lp + "q"], w[lp + "k"] = torch.zeros_like(w[lp + "q"]), torch.zeros_like(w[lp + "k"])
    w[lp + "q"][0], w[lp + "q"][8], w[lp + "k"][0] = b * 3, b * 3, a * 3
    w[lp + "temp"] = torch.ones(2, dtype=O.DT)
    w = {k: v.to(torch.bfloat16).to(O.DT) for k, v in w.items()}
    O.write_model(str(tmp_path), cfg, w)
    oracle = O.Oracle(cfg, w)
    base = [t if t != mark else mark + 1 for t in tokens(60, 30, 9)]
    inside, outside = list(base), list(base)
    inside[59 - 19] = mark        # position 40: the last one position 59 still sees
    outside[59 - 20] = mark       # position 39: the first one it does not
    wi, wo = oracle.forward(inside).numpy(), oracle.forward(outside).numpy()
    assert err(wi[59:], wo[59:]) > 0.1
    for kind in ("f32", "bf16"):
        m = open_model(S, str(tmp_path), kind)
        for seq, want in ((inside, wi), (outside, wo)):
            got = m.step([(0, seq, [58, 59])])
            check(got, want[58:], kind, "prompt rows")
            m.release(0)
            m.step([(0, seq[:59], [])])
            got = m.step([(0, seq[59:], [0])])
            check(got, want[59:], kind, "single token")
            m.release(0)
        m.close()


def test_a_far_key_decides_the_logits_of_a_latent_layer(S, tmp_path):
    """one latent layer, 600 positions: the token `mark` at position 3 takes the softmax of the last query; without it the logits
    are others"""
    cfg, w = O.random_model(seed=6, width=32, vocab=30, layers=[lat(2, 8, 4, 8, 16, 24, scale=3.0, ff=None)])
    mark, mp = 7, "l0.mix."
    h = O.layer_norm(w["embed"], w["l0.norm1"], 1e-5)
    rest = h[[i for i in range(30) if i != mark]]
    a = torch.linalg.lstsq(torch.cat([rest, h[mark:mark + 1] * 8]), torch.cat([torch.zeros(29, 1, dtype=O.DT), torch.full((1, 1), 8.0, dtype=O.DT)])).solution[:, 0]
    b = torch.linalg.lstsq(h, torch.ones(30, 1, dtype=O.DT)).solution[:, 0]
    w[mp + "dkv"][0] = a * 6                       # the first latent column belongs to the marked token
    w[mp + "dq"][0] = b * 6                        # the first query column to everybody
    w[mp + "uk"], w[mp + "uq"] = torch.zeros_like(w[mp + "uk"]), torch.zeros_like(w[mp + "uq"])
    w[mp + "uk"][0, 0] = w[mp + "uk"][8, 0] = w[mp + "uq"][0, 0] = w[mp + "uq"][12, 0] = 1.0
    w = {k: v.to(torch.bfloat16).to(O.DT) for k, v in w.items()}
    O.write_model(str(tmp_path), cfg, w)
    oracle = O.Oracle(cfg, w)
    without = [t if t != mark else mark + 1 for t in tokens(600, 30, 11)]
    marked = list(without)
    marked[3] = mark
    ww, wm = oracle.forward(without).numpy(), oracle.forward(marked).numpy()
    assert err(wm[599:], ww[599:]) > 0.1
    for kind in ("f32", "bf16"):
        m = open_model(S, str(tmp_path), kind)
        for seq, want in ((marked, wm), (without, ww)):
            check(m.step([(0, seq, [500, 599])]), want[[500, 599]], kind, "prompt rows")
            m.release(0)
            m.step([(0, seq[:599], [])])
            check(m.step([(0, seq[599:], [0])]), want[599:], kind, "single token")
            m.release(0)
        m.close()


def test_refused_configurations(S, models, tmp_path):
    folder, oracle, cfg = models["mix"]

    def refused(change, text):
        c = copy.deepcopy(cfg)
        change(c)
        O.write_model(str(tmp_path), c, oracle.w)
        with pytest.raises(RuntimeError, match=text):
            S.Model(str(tmp_path), dtype=S.F32, max_tokens=64, max_slots=1)
    refused(lambda c: c["layers"][1].update(type="retention"), "not part of this family")
    refused(lambda c: c["layers"][0]["mixer"].update(kv_rank=23), "kv_from")
    refused(lambda c: c["layers"][0]["mixer"].update(q_rank=21), "shape")
    refused(lambda c: c["layers"][3]["mixer"]["right"].update(conv=4), "shape")


def test_greedy_generation_through_the_scheduler(S, models):
    """six requests on two slots with an end token, prompts fed in portions of 16 beside the others' single tokens,
    against greedy decoding with the oracle"""
    folder, oracle, cfg = models["mix"]
    V = cfg["vocab"]
    prompts = [tokens(n, V, 40 + i) for i, n in enumerate([5, 40, 17, 1, 33, 70])]
    max_new, eos = 12, 7
    want = []
    for p in prompts:
        seq, outp = list(p), []
        for k in range(max_new):
            nxt = int(oracle.forward(seq)[-1].argmax())
            if k > 0 and nxt == eos:
                break
            outp.append(nxt)
            seq.append(nxt)
        want.append(outp)
    m = open_model(S, folder, "f32", max_tokens=64 * 6, slots=2)
    outs, steps = m.generate(prompts, max_new=max_new, eos_id=eos, chunk=16)
    assert steps > max_new
    assert outs == want
    assert m.pages_free == m.pages_total
    m.close()
