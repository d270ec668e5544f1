"""Each kernel (or kernel option) that the Mazotar family brought to include/b200_serve.h, alone, against the plain functions
of mazotar_oracle.py (or a line of torch): the embedding into several streams, the streams' update with the norm that follows,
norms over whole query / key rows with the query temperature (and queries only, and rotated), paged attention with a distance
bias and a learned sink (row, group and tile kernels; split contexts; masks; keys on both sides of a bucket's edge made to stand
out), the matrix memory (walk and chunk form, stale states, gates that saturate), the weighted head norm with a sigmoid gate, the
sigmoid router with a shared expert's gate, weighted dispatch, scaled gathering and row scales in the grouped product."""
import ctypes as C
import math

import pytest
import torch

import mazotar_oracle as O

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def S(pkg):
    if not torch.cuda.is_available():
        pytest.fail("no CUDA device: the library has no CPU path")
    return pkg.serve


_alive = []


def dev(t, dtype=None):
    t = torch.as_tensor(t).cuda()
    t = t.to(dtype).contiguous() if dtype is not None else t.contiguous()
    _alive.append(t)
    return t


def f32(t):
    return dev(t, torch.float32)


def ints(a):
    return dev(torch.as_tensor(a, dtype=torch.int32))


def empty(*shape, dtype=torch.float32, fill=float("nan")):
    t = torch.full(shape, fill, dtype=dtype, device="cuda")
    _alive.append(t)
    return t


@pytest.fixture(autouse=True)
def _drop_device_tensors():
    yield
    torch.cuda.synchronize()
    _alive.clear()


def tdt(S, code):
    return torch.bfloat16 if code == S.BF16 else torch.float32


def code_of(S, kind):
    return S.BF16 if kind == "bf16" else S.F32


def rel(got, want):
    return float((got.double().cpu() - want.double()).abs().max() / want.double().abs().max().clamp_min(1e-30))


def sync_ok(rc):
    assert rc == 0, f"rc={rc}"
    torch.cuda.synchronize()


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rounded(t, kind):
    return t.to(torch.bfloat16).double() if kind == "bf16" else t.float().double()


def ptr(t):
    return t.data_ptr() if t is not None else None


def paged(S, code, rows, PR, seed):
    """rows: list of dicts slot -> [n, units, d] that share one page table; scatters them into shuffled pages. Rows nobody owns
    hold large values that would dominate if they were read."""
    first = rows[0]
    max_pages = max((len(x) + PR - 1) // PR for x in first.values())
    total = len(first) * max_pages + 3
    order = torch.randperm(total, generator=gen(seed)).tolist()
    table = torch.zeros(len(first), max_pages, dtype=torch.int32)
    pools = [torch.full((total * PR, *next(iter(r.values())).shape[1:]), 300.0) for r in rows]
    for b in first:
        for i in range((len(first[b]) + PR - 1) // PR):
            pg = order.pop()
            table[b, i] = pg
            n = min(PR, len(first[b]) - i * PR)
            for pool, r in zip(pools, rows):
                pool[pg * PR: pg * PR + n] = r[b][i * PR: i * PR + n]
    return [dev(p, tdt(S, code)) for p in pools], dev(table), max_pages


# ---------------------------------------------------------------------------------------------------------------
# streams
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("streams,width", [(1, 8), (2, 64), (3, 37), (5, 130)])
def test_embedding_into_streams(S, kind, streams, width):
    """sinusoids at positions up to a million (double angles), an odd width; without the sinusoids the scaled rows alone"""
    table = rounded(torch.randn(11, width, generator=gen(width)), kind)
    ids, pos = [3, 0, 10, 3, 7], [0, 1, 777, 100003, 1000000]
    pe = torch.zeros(5, width, dtype=O.DT)
    for r, p in enumerate(pos):
        for c in range(width):
            ang = p * 10000.0 ** (-2.0 * (c // 2) / width)
            pe[r, c] = math.cos(ang) if c % 2 else math.sin(ang)
    turns = dev(torch.tensor([10000.0 ** (-2.0 * i / width) / math.pi for i in range((width + 1) // 2)], dtype=torch.float64))
    tab = dev(table, tdt(S, code_of(S, kind)))
    for with_pos in (True, False):
        out = empty(5, streams, width)
        sync_ok(S.lib().b200_embed_streams(ptr(ints(ids)), ptr(ints(pos)), ptr(tab), 1.75, ptr(turns) if with_pos else None, ptr(out), streams, 5, width,
                                           code_of(S, kind), None))
        want = table[ids] * 1.75 + (pe if with_pos else 0)
        for s in range(streams):
            assert float((out[:, s].double().cpu() - want).abs().max()) < 2e-6


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("streams,width,top", [(1, 36, 1), (2, 64, 3), (3, 2048, 2), (4, 4096, 16), (4, 37, 1), (2, 8192, 1), (5, 100, 4), (16, 1, 2), (4, 9000, 1), (3, 1028, 0)])
def test_update_of_all_streams_and_the_norm_that_follows(S, kind, streams, width, top):
    T, g, eps = 5, gen(streams * width), 1e-4
    x = torch.randn(T, streams, width, generator=g)
    mix, w_out, w_in = torch.randn(streams, streams, generator=g), torch.randn(streams, generator=g), torch.randn(streams, generator=g)
    y1, y2, gate = torch.randn(T, width, generator=g), torch.randn(T, width, generator=g), torch.rand(T, generator=g)
    eo = torch.randn(T * max(top, 1), width, generator=g)
    dest = torch.randperm(T * max(top, 1), generator=g).view(T, -1).to(torch.int32)
    if top > 1:
        dest[1, 0] = -1     # an expert without a row adds nothing
    wt = torch.rand(T, max(top, 1), generator=g)
    w = torch.randn(width, generator=g)
    code = code_of(S, kind)

    def call(**kw):
        a = S.HyperResidualArgs(streams=streams, eps=eps, out_dtype=code, n_rows=T, width=width, top=top)
        keep = {}
        for k, v in kw.items():
            if isinstance(v, torch.Tensor):
                keep[k] = v if v.is_cuda else dev(v)
                v = keep[k].data_ptr()
            setattr(a, k, v)
        sync_ok(S.lib().b200_hyper_residual(C.byref(a), None))

    def plain(y, reads):
        n = torch.einsum("sr,tsd->trd", mix.double(), x.double()) + w_out.double()[None, :, None] * y[:, None, :]
        u = torch.einsum("s,tsd->td", reads, n)
        return n, u
    rows = torch.zeros(T, width, dtype=O.DT)
    weighted = torch.zeros(T, width, dtype=O.DT)
    for t in range(T):
        for k in range(top):
            if dest[t, k] >= 0:
                rows[t] += eo[dest[t, k]].double()
                weighted[t] += eo[dest[t, k]].double() * wt[t, k].double()
    tol = 1e-5 if kind == "f32" else 6e-3
    cases = [(dict(y1=y1), y1.double()), (dict(y2=y2, gate2=gate), y2.double() * gate.double()[:, None])]
    if top:
        cases += [(dict(expert_out=eo, dest=dest), rows), (dict(expert_out=eo, dest=dest, weight=wt, y1=y1, y2=y2), weighted + y1.double() + y2.double())]
    for kw, y in cases:
        xd, out, total = f32(x), empty(T, width, dtype=tdt(S, code)), empty(T, width)
        call(x=xd, mix=mix, w_out=w_out, w_in=w_in, w=w, out=out, **kw)
        n, u = plain(y, w_in.double())
        assert rel(xd, n) < 1e-5
        assert rel(out, O.rms_norm(u, w.double(), eps)) < tol
        xd = f32(x)
        call(x=xd, mix=mix, w_out=w_out, sum_out=total, **kw)      # the sum of the new streams, nothing normed
        n, u = plain(y, torch.ones(streams, dtype=O.DT))
        assert rel(xd, n) < 1e-5 and rel(total, u) < 1e-5
        xd = f32(x)
        call(x=xd, mix=mix, w_out=w_out, **kw)                     # update only
        assert rel(xd, n) < 1e-5
    # reading only: first norm, listed rows, nothing changed
    xd, out = f32(x), empty(T, width, dtype=tdt(S, code))
    call(x=xd, w_in=w_in, w=w, out=out)
    assert rel(out, O.rms_norm(torch.einsum("s,tsd->td", w_in.double(), x.double()), w.double(), eps)) < tol
    call(x=xd, rows=ints([4, 0, 2, 2, 1]), w=w, out=out)
    assert rel(out, O.rms_norm(x.double().sum(1)[[4, 0, 2, 2, 1]], w.double(), eps)) < tol
    assert torch.equal(xd.cpu(), x)


def test_stream_arguments_that_do_not_fit(S):
    a = S.HyperResidualArgs(x=1, streams=2, n_rows=0, width=8, y1=1)
    assert S.lib().b200_hyper_residual(C.byref(a), None) != 0        # an addend without a mixing matrix
    a = S.HyperResidualArgs(x=1, streams=17, n_rows=0, width=8)
    assert S.lib().b200_hyper_residual(C.byref(a), None) != 0
    a = S.HyperResidualArgs(x=1, streams=2, n_rows=0, width=8, w=1)
    assert S.lib().b200_hyper_residual(C.byref(a), None) != 0        # a norm without an output


# ---------------------------------------------------------------------------------------------------------------
# query / key rows
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("H,G,d,dv,rot", [(4, 2, 16, 24, 0), (3, 1, 5, 7, 0), (16, 8, 128, 128, 0), (64, 16, 128, 64, 0), (4, 4, 12, 9, 8), (6, 2, 10, 6, 10), (40, 40, 130, 3, 0)])
def test_norms_over_whole_query_and_key_rows(S, kind, H, G, d, dv, rot):
    """register, two-pass and rotated kernels: normed keys and projected values land in the pages, queries carry the temperature of
    their position; the same queries when the layer has no keys of its own"""
    code, g, PR, eps = code_of(S, kind), gen(H + d), 16, 1e-3
    pos, slot, every, coef = [0, 1, 40, 41, 99], [0, 0, 1, 1, 0], 7, 0.6
    T, nq, nk, nv = 5, H * d, G * d, G * dv
    ld = nq + nk + nv + 8
    ld += -ld % 4
    proj = torch.randn(T, ld, generator=g)
    qn, kn = torch.randn(nq, generator=g), torch.randn(nk, generator=g)
    kc = {b: torch.zeros(112, G, d) for b in (0, 1)}
    vc = {b: torch.zeros(112, G, dv) for b in (0, 1)}
    (kp, vp), table, mp = paged(S, code, [kc, vc], PR, 1)
    ang = torch.tensor(pos, dtype=O.DT)[:, None] * torch.tensor([10.0 ** (-m) for m in range(max(rot // 2, 1))], dtype=O.DT)
    cs, sn = f32(torch.cos(ang)), f32(torch.sin(ang))

    def turn(y):
        if not rot:
            return y
        P = rot // 2
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        a, b = y[..., :P], y[..., P:rot]
        return torch.cat([a * c - b * s, b * c + a * s, y[..., rot:]], -1)
    pd = proj.double()
    temp = torch.tensor([1 + coef * math.log((p + 1) // every + 1) for p in pos], dtype=O.DT)
    q = turn(O.rms_norm(pd[:, :nq], qn.double(), eps).view(T, H, d)) * temp[:, None, None]
    k = turn(O.rms_norm(pd[:, nq:nq + nk], kn.double(), eps).view(T, G, d))
    v = pd[:, nq + nk:nq + nk + nv].view(T, G, dv)
    tol = 2e-6 if kind == "f32" else 5e-3
    prd = f32(proj)
    for own in (True, False):
        qo = empty(T, nq, dtype=tdt(S, code))
        before = kp.clone()
        a = S.QkPrepareArgs(proj=ptr(prd), ld_proj=ld, q_norm=ptr(f32(qn)), k_norm=ptr(f32(kn)) if own else None, eps=eps, q_out=ptr(qo), pages=ptr(table),
                            max_pages=mp, page_rows=PR, slot=ptr(ints(slot)), pos=ptr(ints(pos)), start=ptr(ints(pos)), n_tokens=T, heads=H, kv_heads=G,
                            dim=d, dtype=code, norm_rows=1, temp_coef=coef, temp_every=every, rot_dims=rot, rot_layout=S.ROPE_HALF)
        if rot:
            a.cos, a.sin = ptr(cs), ptr(sn)
        if own:
            a.k_pool, a.v_pool, a.v_heads, a.vdim, a.v_off = ptr(kp), ptr(vp), G, dv, nq + nk
        sync_ok(S.lib().b200_qk_prepare(C.byref(a), None))
        assert rel(qo.view(T, H, d), q) < tol
        if not own:
            assert torch.equal(kp, before)
            continue
        for t in range(T):
            row = int(table[slot[t], pos[t] // PR]) * PR + pos[t] % PR
            assert rel(kp[row], k[t]) < tol and rel(vp[row], v[t]) < tol
    kn2 = a.k_pool
    a.conv_w, a.taps = 1, 2
    assert S.lib().b200_qk_prepare(C.byref(a), None) != 0 and kn2 is None       # no convolution beside row norms


def test_temperature_beside_norms_per_head(S):
    """the temperature in the per-head kernel (no norm at all: the plain scatter must not swallow it)"""
    T, H, G, d, PR = 3, 2, 1, 8, 16
    g = gen(4)
    proj, pos = torch.randn(T, (H + G) * d, generator=g), [5, 6, 30]
    for norm in (None, torch.randn(d, generator=g)):
        kp, qo, table = empty(4 * PR, G, d), empty(T, H * d), ints([[0, 1, 2, 3]])
        a = S.QkPrepareArgs(proj=ptr(f32(proj)), ld_proj=(H + G) * d, q_norm=ptr(f32(norm)) if norm is not None else None, eps=1e-5, q_out=ptr(qo), k_pool=ptr(kp),
                            pages=ptr(table), max_pages=4, page_rows=PR, slot=ptr(ints([0, 0, 0])), pos=ptr(ints(pos)), start=ptr(ints(pos)), n_tokens=T,
                            heads=H, kv_heads=G, dim=d, dtype=S.F32, temp_coef=0.5, temp_every=3)
        sync_ok(S.lib().b200_qk_prepare(C.byref(a), None))
        q = proj[:, :H * d].double().view(T, H, d)
        if norm is not None:
            q = O.rms_norm(q, norm.double(), 1e-5)
        assert rel(qo.view(T, H, d), q * torch.tensor([1 + 0.5 * math.log((p + 1) // 3 + 1) for p in pos], dtype=O.DT)[:, None, None]) < 2e-6
        assert rel(kp[pos], proj[:, H * d:].double().view(T, G, d)) < 2e-6


# ---------------------------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------------------------
def plain_attention(q, k, v, pos, scale, table, sink, window=0, cap=0.0):
    """q [T, H, d] at positions pos of ONE sequence whose keys start at position 0; table [H, n] per distance or None, sink [H] or None"""
    H, G = q.shape[1], k.shape[1]
    back = torch.tensor(pos)[:, None] - torch.arange(len(k))[None, :]
    s = torch.einsum("thd,nhd->htn", q, k.repeat_interleave(H // G, 1)) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    if table is not None:
        s = s + table[:, back.clamp(0, table.shape[1] - 1)]
    ok = (back >= 0) & (back < window) if window else back >= 0
    s = s.masked_fill(~ok, float("-inf"))
    p = O.sink_softmax(s, sink) if sink is not None else torch.softmax(s, -1)
    return torch.einsum("htn,nhc->thc", p, v.repeat_interleave(H // G, 1))


ATT_SHAPES = [  # heads, kv, dim, vdim, distances, window
    (4, 2, 16, 24, 37, 0),       # padded tiles
    (3, 3, 10, 6, 5, 0),         # nothing a multiple of 8: the row kernel in both types
    (5, 1, 6, 7, 1, 0),          # one number for every distance
    (6, 2, 64, 72, 130, 0),      # three heads per key head, padded values
    (8, 8, 64, 64, 200, 0),      # an exact tile
    (8, 4, 128, 128, 90, 0),     # an exact tile
    (4, 1, 128, 256, 500, 0),    # wide values
    (8, 2, 64, 128, 33, 0),
    (4, 2, 72, 40, 60, 50),      # with a window
    (2, 2, 128, 128, 60, 90),
    (2, 1, 200, 200, 300, 0),    # wider keys than the tiles take
    (16, 2, 32, 16, 64, 0),      # eight heads per key head
]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("shape", ATT_SHAPES)
def test_attention_with_distance_bias_and_sinks(S, shape, kind):
    """two sequences in one batch: a prompt portion of 150 tokens behind 330 cached ones, and a single token at position 77; then the
    last tokens of both alone (with and without a workspace for split contexts). In one query the keys on both sides of a step in
    the table, the oldest key and one at a page's edge are made to stand out with values of their own."""
    H, G, d, dv, n_dist, win = shape
    code, g, PR = code_of(S, kind), gen(sum(shape)), 64
    n0, new0, n1 = 480, 150, 78
    scale = 1.0 / math.sqrt(d)
    k = {0: rounded(torch.randn(n0, G, d, generator=g), kind), 1: rounded(torch.randn(n1, G, d, generator=g), kind)}
    v = {0: rounded(torch.randn(n0, G, dv, generator=g), kind), 1: rounded(torch.randn(n1, G, dv, generator=g), kind)}
    pos, slot = list(range(n0 - new0, n0)) + [n1 - 1], [0] * new0 + [1]
    q = rounded(torch.randn(new0 + 1, H, d, generator=g), kind)
    table, sink = torch.randn(H, n_dist, generator=g), torch.randn(H, generator=g) + 1
    star = 100                       # the query at position 430
    at = pos[star]
    marks = [j for j in {at, at - 1, at - n_dist + 1, at - n_dist, 0, 63, 64, 127, at - win + 1, at - win} if 0 <= j <= at]
    for j in marks:
        for kg in range(G):
            k[0][j, kg] = rounded(q[star, kg * (H // G)] * (3.0 / scale / float((q[star, kg * (H // G)] ** 2).sum())), kind)
        v[0][j] += 6.0
    v = {b: rounded(x, kind) for b, x in v.items()}
    (kp, vp), pages, mp = paged(S, code, [k, v], PR, 2)
    td, sd = f32(table), f32(sink)
    ws = empty(64 << 18)
    tol = 3e-6 if kind == "f32" else 1.5e-2

    def run(rows, use_table, use_sink, longest, workspace=True, cap=0.0):
        qd, out = dev(q[rows], tdt(S, code)), empty(len(rows), H * dv, dtype=tdt(S, code))
        a = S.PagedAttentionArgs(q=ptr(qd), out=ptr(out), k_pool=ptr(kp), v_pool=ptr(vp), pages=ptr(pages), max_pages=mp, page_rows=PR,
                                 slot=ptr(ints([slot[r] for r in rows])), pos=ptr(ints([pos[r] for r in rows])), n_tokens=len(rows), heads=H, kv_heads=G, dim=d,
                                 vdim=dv, scale=scale, softcap=cap, dtype=code, longest_entry=longest, longest_context=n0, window=win)
        if workspace:
            a.workspace, a.workspace_bytes = ptr(ws), ws.numel() * 4
        if use_table:
            a.dist_bias, a.dist_n = ptr(td), n_dist
        if use_sink:
            a.sink = ptr(sd)
        sync_ok(S.lib().b200_paged_attention(C.byref(a), None))
        want = torch.cat([plain_attention(q[[r]], k[slot[r]], v[slot[r]], [pos[r]], scale, table.double() if use_table else None, sink.double() if use_sink else None,
                                          win, cap) for r in rows])
        assert rel(out.view(len(rows), H, dv), want) < tol, (use_table, use_sink, longest, workspace, cap)
    everything = list(range(new0 + 1))
    run(everything, True, True, new0)
    run(everything, True, False, new0)
    run(everything, False, True, new0)
    run([star, new0 - 1, new0][1:], True, True, 1)
    run([star], True, True, 1)
    run([star], True, True, 1, workspace=False)
    run([0, star, new0 - 1, new0], True, True, 2, cap=3.0)      # a cap under the bias: the row kernel


def test_the_standing_out_keys_really_do(S):
    """sensitivity of the test above: a table that is one distance off, a sink left out or a scaled bias moves the star query's output
    by far more than the tolerance"""
    H, G, d, n_dist = 4, 2, 16, 37
    g = gen(1)
    q, k, v = torch.randn(1, H, d, generator=g).double(), torch.randn(431, G, d, generator=g).double(), torch.randn(431, G, 8, generator=g).double()
    table, sink = torch.randn(H, n_dist, generator=g).double(), torch.randn(H, generator=g).double() + 1
    for j in (430, 394, 393, 0):
        for kg in range(G):
            k[j, kg] = q[0, kg * 2] * (3.0 / 0.25 / float((q[0, kg * 2] ** 2).sum()))
        v[j] += 6.0
    base = plain_attention(q, k, v, [430], 0.25, table, sink)
    off = torch.cat([table[:, :1], table[:, :-1]], 1)
    for other in (plain_attention(q, k, v, [430], 0.25, off, sink), plain_attention(q, k, v, [430], 0.25, table, None),
                  plain_attention(q, k, v, [430], 0.25, table * 0.25, sink)):
        assert rel(other, base) > 2e-2


def test_one_key_tile_and_rows_that_change_sequences(S):
    """prompts shorter than one key tile, several sequences inside one tile of rows, each on pages of its own"""
    g = gen(9)
    for H, G, d, dv in ((4, 2, 64, 64), (4, 2, 128, 128), (4, 4, 40, 24), (2, 1, 64, 80), (2, 2, 128, 256)):
        lens = [3, 50, 17, 64, 1, 33]
        k = {b: rounded(torch.randn(n, G, d, generator=g), "bf16") for b, n in enumerate(lens)}
        v = {b: rounded(torch.randn(n, G, dv, generator=g), "bf16") for b, n in enumerate(lens)}
        (kp, vp), pages, mp = paged(S, S.BF16, [k, v], 16, 3)
        pos, slot = [p for n in lens for p in range(n)], [b for b, n in enumerate(lens) for _ in range(n)]
        q = rounded(torch.randn(len(pos), H, d, generator=g), "bf16")
        table, sink = torch.randn(H, 20, generator=g), torch.randn(H, generator=g)
        want = torch.cat([plain_attention(q[[r for r in range(len(pos)) if slot[r] == b]], k[b], v[b], list(range(n)), 0.2, table.double(), sink.double())
                          for b, n in enumerate(lens)])
        for turn in range(4):
            out = empty(len(pos), H * dv, dtype=torch.bfloat16)
            a = S.PagedAttentionArgs(q=ptr(dev(q, torch.bfloat16)), out=ptr(out), k_pool=ptr(kp), v_pool=ptr(vp), pages=ptr(pages), max_pages=mp, page_rows=16,
                                     slot=ptr(ints(slot)), pos=ptr(ints(pos)), n_tokens=len(pos), heads=H, kv_heads=G, dim=d, vdim=dv, scale=0.2, dtype=S.BF16,
                                     longest_entry=64, longest_context=64, sink=ptr(f32(sink)), dist_bias=ptr(f32(table)), dist_n=20)
            sync_ok(S.lib().b200_paged_attention(C.byref(a), None))
            assert rel(out.view(len(pos), H, dv), want) < 1.5e-2, (H, G, d, dv, turn)


def test_attention_options_that_exclude_each_other(S):
    base = dict(q=1, out=1, k_pool=1, v_pool=1, pages=1, slot=1, pos=1, n_tokens=0, heads=2, kv_heads=1, dim=8, vdim=8, page_rows=64, dtype=S.F32)
    for bad in (dict(sink=1, sigmoid_weights=1), dict(sink=1, denom_bias=1.0), dict(dist_bias=1, dist_n=0), dict(dist_bias=1, dist_n=4, head_mix=1)):
        assert S.lib().b200_paged_attention(C.byref(S.PagedAttentionArgs(**base, **bad)), None) != 0, bad


# ---------------------------------------------------------------------------------------------------------------
# matrix memory
# ---------------------------------------------------------------------------------------------------------------
MEM_SHAPES = [  # heads, dim, vdim
    (2, 16, 32), (3, 5, 7), (1, 1, 1), (2, 64, 64), (4, 48, 80), (2, 128, 256), (1, 200, 130), (2, 33, 65), (1, 256, 64), (1, 300, 40),
]


@pytest.mark.parametrize("chunked", [0, 1])
@pytest.mark.parametrize("shape", MEM_SHAPES)
@pytest.mark.parametrize("gates", ["open", "forgetting", "shut"])
def test_matrix_memory_over_several_calls(S, shape, chunked, gates):
    """three unequal entries over three calls above stale memories; the second call continues two sequences and starts one anew in a
    used slot. Gates: mostly open; forget gates near zero with inputs that win at once; input gates far below the maximum (the
    denominator rests on its floor)"""
    H, d, p = shape
    g, cap = gen(sum(shape) + chunked), 9.0
    nq, nv = H * d, H * p
    offs = dict(q_off=0, k_off=nq, v_off=2 * nq, i_off=2 * nq + nv, f_off=2 * nq + nv + H)
    ld = 2 * nq + nv + 2 * H
    ld += -ld % 4
    shift = {"open": (0.0, 4.0), "forgetting": (2.0, -6.0), "shut": (-8.0, 3.0)}[gates]
    ib, fb = torch.randn(H, generator=g) + shift[0], torch.randn(H, generator=g) + shift[1]
    per = int(S.lib().b200_mlstm_norm_floats(d, p))
    state, norm = empty(4, H, d, p, fill=7.0), empty(4, H, per, fill=3.0)
    seqs = {b: torch.zeros(0, ld) for b in range(4)}
    scale = d ** -0.5
    tol = 2e-5 if not chunked else 4e-3
    # (slot, new tokens, starts anew) of each call, in batch order
    calls = [[(2, 130, True), (0, 5, True), (3, 1, True)], [(3, 200, False), (2, 1, False), (0, 70, True)], [(0, 1, False), (1, 2, True), (3, 64, False), (2, 300, False)]]
    for entries in calls:
        new = {b: torch.randn(n, ld, generator=g) for b, n, _ in entries}
        row, rows, lens, slot, pos = 0, [], [], [], []
        for b, n, anew in entries:
            if anew:
                seqs[b] = torch.zeros(0, ld)
            rows.append(row); lens.append(n)
            slot += [b] * n; pos += list(range(len(seqs[b]), len(seqs[b]) + n))
            seqs[b] = torch.cat([seqs[b], new[b]])
            row += n
        proj, out = f32(torch.cat([new[b] for b, _, _ in entries])), empty(row, nv)
        need = int(S.lib().b200_mlstm_workspace_bytes(row, len(entries), H, d, p))
        ws = empty(max(need, 256) // 4 + 1)
        a = S.MlstmArgs(proj=ptr(proj), ld_proj=ld, i_bias=ptr(f32(ib)), f_bias=ptr(f32(fb)), gate_cap=cap, q_scale=scale, state=ptr(state), norm=ptr(norm),
                        out=ptr(out), ent_row=ptr(ints(rows)), ent_len=ptr(ints(lens)), slot=ptr(ints(slot)), pos=ptr(ints(pos)), n_entries=len(entries),
                        n_tokens=row, heads=H, dim=d, vdim=p, longest_entry=max(lens), chunked=chunked, workspace=ptr(ws), workspace_bytes=need, **offs)
        sync_ok(S.lib().b200_mlstm(C.byref(a), None))
        for (b, n, _), r in zip(entries, rows):
            u = seqs[b].double()
            T = len(u)
            li = O.capped(u[:, offs["i_off"]:offs["i_off"] + H] + ib.double(), cap)
            lf = torch.nn.functional.logsigmoid(O.capped(u[:, offs["f_off"]:offs["f_off"] + H] + fb.double(), cap))
            want = O.mlstm_memory(u[:, :nq].view(T, H, d) * scale, u[:, nq:2 * nq].view(T, H, d), u[:, 2 * nq:2 * nq + nv].view(T, H, p), li, lf)[T - n:].reshape(n, nv)
            got = out[r:r + n].double().cpu()
            assert torch.isfinite(got).all()
            # against a row's own size (denominators that nearly cancel make single rows large), but not below a fiftieth of the largest
            e = (got - want).abs().amax(1) / want.abs().amax(1).clamp_min(float(want.abs().max()) / 50)
            assert float(e.max() if not chunked else e.quantile(0.95)) < tol * (30 if not chunked else 4), float(e.max())
            assert float(e.median()) < tol


def test_memory_arguments_that_do_not_fit(S):
    a = S.MlstmArgs(proj=1, i_bias=1, f_bias=1, gate_cap=0.0, state=1, norm=16, out=1, ent_row=1, ent_len=1, slot=1, pos=1, heads=1, dim=1, vdim=1)
    assert S.lib().b200_mlstm(C.byref(a), None) != 0
    a.gate_cap, a.dim = 1.0, 513
    assert S.lib().b200_mlstm(C.byref(a), None) != 0


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("H,p", [(2, 64), (3, 7), (1, 256), (4, 500), (2, 520), (5, 1)])
def test_head_norm_with_weight_and_gate(S, kind, H, p):
    T, g, eps = 6, gen(H + p), 1e-3
    o, z, w = torch.randn(T, H * p, generator=g), torch.randn(T, H * p + 12, generator=g), torch.randn(H * p, generator=g)
    code = code_of(S, kind)
    od, zd, wd = f32(o), f32(z), f32(w)
    for off in (0, 4, 3):
        zz = z[:, off:off + H * p].double()
        n = O.unit_rms(o.double().view(T, H, p), eps).view(T, H * p)
        for weight, sig in ((wd, 1), (None, 0), (wd, 0), (None, 1)):
            out = empty(T, H * p, dtype=tdt(S, code))
            sync_ok(S.lib().b200_head_rms_gate(ptr(od), zd.data_ptr() + 4 * off, H * p + 12, ptr(weight), sig, ptr(out), T, H, p, eps, code, None))
            want = n * (w.double() if weight is not None else 1) * (torch.sigmoid(zz) if sig else O.silu(zz))
            assert rel(out, want) < (2e-6 if kind == "f32" else 5e-3)


# ---------------------------------------------------------------------------------------------------------------
# experts
# ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("E,top,gates,width", [(8, 2, 1, 64), (1, 1, 0, 7), (5, 5, 1, 33), (16, 3, 1, 2048), (40, 4, 2, 130), (130, 16, 0, 96)])
def test_sigmoid_router(S, kind, E, top, gates, width):
    T, g = 9, gen(E + width)
    h = rounded(torch.randn(T, width, generator=g), kind)
    w = torch.randn(E + gates, width, generator=g) * (2.0 / math.sqrt(width))
    chosen, weight, gv = empty(T, top, dtype=torch.int32, fill=-7), empty(T, top), empty(T, max(gates, 1))
    sync_ok(S.lib().b200_moe_route_sigmoid(ptr(dev(h, tdt(S, code_of(S, kind)))), code_of(S, kind), ptr(f32(w)), T, width, E, top, gates, ptr(chosen), ptr(weight),
                                           ptr(gv) if gates else None, None))
    z = h @ w.double().T
    want, ww = O.route(z[:, :E], top)
    assert torch.equal(chosen.cpu().long(), want)
    assert float((weight.double().cpu() - ww).abs().max()) < 2e-6
    if gates:
        assert float((gv.double().cpu() - torch.sigmoid(z[:, E:])).abs().max()) < 2e-6


def test_router_ties_and_saturated_scores(S):
    """equal logits: the lower index; logits whose sigmoids round to one are still told apart"""
    h = torch.zeros(3, 4)
    h[1, 0], h[2, 1] = 1.0, 1.0
    w = torch.zeros(6, 4)
    w[:, 0] = torch.tensor([1.0, 2.0, 2.0, 0.0, 2.0, 1.0])
    w[:, 1] = torch.tensor([40.0, 50.0, 60.0, 70.0, 45.0, 55.0])
    chosen, weight = empty(3, 3, dtype=torch.int32, fill=-7), empty(3, 3)
    sync_ok(S.lib().b200_moe_route_sigmoid(ptr(f32(h)), S.F32, ptr(f32(w)), 3, 4, 6, 3, 0, ptr(chosen), ptr(weight), None, None))
    assert chosen.cpu().tolist() == [[0, 1, 2], [1, 2, 4], [3, 2, 5]]
    assert weight.cpu().tolist()[0] == [0.5, 0.5, 0.5] and weight.cpu().tolist()[2] == [1.0, 1.0, 1.0]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width,ff,E,top", [(64, 32, 5, 2), (37, 9, 3, 3), (128, 128, 4, 1)])
def test_experts_that_read_their_input_times_its_weight(S, kind, width, ff, E, top):
    """routing, weighted dispatch, the grouped product with row scales against gathered rows scaled one by one, and both against the
    plain statement"""
    T, g, code = 70, gen(width + ff), code_of(S, kind)
    h = rounded(torch.randn(T, width, generator=g), kind)
    W = {}
    for e in range(E):
        W["e%d.gate" % e], W["e%d.up" % e] = rounded(torch.randn(ff, width, generator=g) / math.sqrt(width), kind), rounded(torch.randn(ff, width, generator=g) / math.sqrt(width), kind)
        W["e%d.down" % e] = rounded(torch.randn(width, ff, generator=g) / math.sqrt(ff), kind)
    chosen, wt = O.route(torch.randn(T, E, generator=g).double(), top)
    cd, wd = ints(chosen.int()), f32(wt)
    off, src, dest, roww = empty(E + 1, dtype=torch.int32, fill=-1), empty(T * top, dtype=torch.int32, fill=-1), empty(T, top, dtype=torch.int32, fill=-1), empty(T * top)
    sync_ok(S.lib().b200_moe_dispatch_weighted(ptr(cd), ptr(wd), T, top, E, ptr(off), ptr(src), ptr(dest), ptr(roww), None))
    assert torch.equal(roww.cpu()[dest.cpu().long()], wd.cpu())
    t = tdt(S, code)
    hd = dev(h, t)
    gu = dev(torch.cat([torch.cat([W["e%d.gate" % e], W["e%d.up" % e]]) for e in range(E)]), t)
    want = torch.zeros(T, top, ff, dtype=O.DT)
    for i in range(T):
        for k in range(top):
            x, e = h[i] * wt[i, k], int(chosen[i, k])
            want[i, k] = O.silu(W["e%d.gate" % e] @ x) * (W["e%d.up" % e] @ x)
    rows = empty(T * top, width, dtype=t)
    sync_ok(S.lib().b200_gather_rows_scaled(ptr(hd), ptr(src), ptr(roww), ptr(rows), T * top, width, code, None))
    assert rel(rows[dest.long().view(-1)].view(T, top, width), h[:, None, :] * wt[..., None]) < (1e-6 if kind == "f32" else 5e-3)
    for scaled in (True, False):
        act = empty(T * top, ff, dtype=t)
        a = S.GemmGroupedArgs(A=ptr(hd if scaled else rows), lda=width, W=ptr(gu), ldw=width, stride_w=2 * ff * width, C=ptr(act), ldc=ff, group_off=ptr(off), M=T, N=ff,
                              K=width, batch=E, trans_b=1, epi=S.GG_GLU, a_dtype=code, w_dtype=code, c_dtype=code)
        if scaled:
            a.a_rows, a.row_scale = ptr(src), ptr(roww)
        sync_ok(S.lib().b200_gemm_grouped(C.byref(a), None))
        assert rel(act[dest.long().view(-1)].view(T, top, ff), want) < (1e-5 if kind == "f32" else 1.5e-2)
