"""Each kernel (or kernel option) that the Filipel family brought to include/b200_serve.h, alone, against the plain functions
of filipel_oracle.py (or a line of torch): paged attention whose weights are mixed across heads (row kernel with and without
a cluster, prompt tiles in one and in several blocks of rows; keys just inside and just outside the window made to stand
out), per-head temperatures in the unmixed kernels, the state-space recurrence with its carried state (walk and chunk form),
the gated norm in parts, the activation of normed powers, the parallel residual update, the router with groups, the two
low-rank norms with the rotated key part, the layer norm without bias."""
import ctypes as C
import math

import pytest
import torch

import filipel_oracle as O

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


def empty(*shape, dtype=torch.float32, fill=0.0):
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


def plain_mixed(q, k, v, pos, window, scale, temp, talk):
    """q [T, H, d] at positions pos of ONE sequence whose keys k [n, G, d], values v [n, G, dv] start at position 0; talk None:
    the weights as they are"""
    H, G = q.shape[1], k.shape[1]
    kk, vv = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    back = torch.tensor(pos)[:, None] - torch.arange(len(k))[None, :]
    ok = (back >= 0) & (back < window) if window else back >= 0
    s = torch.einsum("thd,nhd->htn", q, kk) * scale * temp[:, None, None]
    p = torch.softmax(s.masked_fill(~ok, float("-inf")), -1)
    if talk is not None:
        p = torch.einsum("hg,gtn->htn", talk, p)
    return torch.einsum("htn,nhc->thc", p, vv)


MIX_SHAPES = [  # heads, kv, dim, vdim, window
    (4, 2, 16, 24, 37),      # two heads per key head; tiles in bfloat16
    (3, 3, 10, 6, 5),        # nothing a multiple of 8: the row kernel in both types
    (5, 1, 6, 7, 0),         # five heads on one key head, odd values, no window
    (8, 1, 64, 56, 70),      # eight heads on one key head
    (4, 1, 72, 40, 33),      # padded score tiles
    (16, 4, 128, 128, 300),  # a context shared by a cluster
    (1, 1, 4, 2, 1),         # one head that only sees itself
    (12, 6, 32, 256, 200),   # wide values
    (40, 20, 24, 16, 90),    # more than 32 heads
    (24, 8, 16, 8, 130),     # three heads per key head
]


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("shape", MIX_SHAPES)
def test_attention_with_weights_mixed_across_heads(S, shape, kind):
    """two sequences in one batch: a prompt portion of 150 tokens behind 330 cached ones, and a single token at position 77. One
    query's keys at the two edges of its window and one far back are made to win its softmax, with values of their own: the
    inside one must count in full, through the mix in every head, the others not at all."""
    H, G, d, dv, win = shape
    code, g, PR = code_of(S, kind), gen(sum(shape)), 64
    n0, new0, n1 = 480, 150, 78
    scale = 1.0 / math.sqrt(d)
    k = {0: rounded(torch.randn(n0, G, d, generator=g), kind), 1: rounded(torch.randn(n1, G, d, generator=g), kind)}
    v = {0: rounded(torch.randn(n0, G, dv, generator=g), kind), 1: rounded(torch.randn(n1, G, dv, generator=g), kind)}
    pos, slot = list(range(n0 - new0, n0)) + [n1 - 1], [0] * new0 + [1]
    q = rounded(torch.randn(len(pos), H, d, generator=g) * 2, kind)
    temp = rounded(1 + torch.randn(H, generator=g) * 0.3, "bf16").abs() + 0.25
    talk = rounded(0.6 * torch.eye(H) + torch.randn(H, H, generator=g) * 0.5, "bf16")
    p = pos[100]
    if win:
        u = torch.zeros(d, dtype=torch.float64)
        u[0] = 1.0
        q[100] = rounded(u * 20.0 / scale / 4.0, kind)
        for j, val, col in ((p - win + 1, 40.0, 0), (p - win, -400.0, 1 % dv), (max(p - win - 130, 0), -400.0, 1 % dv)):
            k[0][j] = rounded(u * 8.0, kind)
            v[0][j] = 0.0
            v[0][j, :, col] = val
    (kp, vp), table, max_pages = paged(S, code, [k, v], PR, 5)
    want = torch.cat([plain_mixed(q[:new0], k[0], v[0], pos[:new0], win, scale, temp, talk),
                      plain_mixed(q[new0:], k[1], v[1], pos[new0:], win, scale, temp, talk)])
    if win > 1:
        assert torch.allclose(want[100, :, 0], 40.0 * talk.sum(1), atol=1.0)   # every head's own weight of that key is one

    def run(qq, sl, ps, longest, with_ws=True):
        T = len(sl)
        out = empty(T, H * dv, fill=float("nan"))
        need = S.lib().b200_mixed_attention_workspace_bytes(T, H, win, max(ps) + 1) if with_ws else 0
        ws = torch.full((max(need, 16),), 255, dtype=torch.uint8, device="cuda")       # not-a-number wherever nothing was written
        _alive.append(ws)
        a = S.PagedAttentionArgs(dev(qq.reshape(T, -1), tdt(S, code)).data_ptr(), out.data_ptr(), kp.data_ptr(), vp.data_ptr(), table.data_ptr(), max_pages,
                                 PR, ints(sl).data_ptr(), ints(ps).data_ptr(), T, H, G, d, dv, scale, 0.0, 0.0, code, longest, max(ps) + 1,
                                 ws.data_ptr() if need else None, need, 0, 1, 1, win, 0, None, f32(temp).data_ptr(), f32(talk).data_ptr())
        sync_ok(S.lib().b200_paged_attention(C.byref(a), None))
        return out.reshape(T, H, dv)

    tol = 2e-2 if kind == "bf16" else 2e-5
    assert rel(run(q, slot, pos, new0), want) < tol                       # the mixed batch
    assert rel(run(q, slot, pos, new0, with_ws=False), want) < 2e-5       # the row kernel on the same batch: fp32 arithmetic
    pick = [100, new0 - 1, new0]                                          # single tokens: the context is shared by a cluster
    assert rel(run(q[pick], [slot[i] for i in pick], [pos[i] for i in pick], 1), want[pick]) < 2e-5


def test_mixed_prompt_rows_in_several_blocks(S):
    """so many heads and so wide a window that the workspace holds a part of the rows at a time (bfloat16 tiles)"""
    H, G, d, dv, win, n = 64, 8, 16, 16, 1000, 1500
    code, g, PR = S.BF16, gen(8), 64
    k = {0: rounded(torch.randn(n, G, d, generator=g), "bf16")}
    v = {0: rounded(torch.randn(n, G, dv, generator=g), "bf16")}
    pos = list(range(n - 900, n))
    q = rounded(torch.randn(900, H, d, generator=g), "bf16")
    temp, talk = torch.ones(H, dtype=torch.float64), rounded(torch.randn(H, H, generator=g) * 0.3, "bf16")
    (kp, vp), table, max_pages = paged(S, code, [k, v], PR, 5)
    need = S.lib().b200_mixed_attention_workspace_bytes(900, H, win, n)
    assert 0 < need < 900 * H * 1152 * 6                                   # less than all rows at once
    ws, out = torch.full((need,), 255, dtype=torch.uint8, device="cuda"), empty(900, H * dv)
    _alive.append(ws)
    a = S.PagedAttentionArgs(dev(q.reshape(900, -1), torch.bfloat16).data_ptr(), out.data_ptr(), kp.data_ptr(), vp.data_ptr(), table.data_ptr(), max_pages,
                             PR, ints([0] * 900).data_ptr(), ints(pos).data_ptr(), 900, H, G, d, dv, 0.25, 0.0, 0.0, code, 900, n, ws.data_ptr(), need,
                             0, 1, 1, win, 0, None, None, f32(talk).data_ptr())
    sync_ok(S.lib().b200_paged_attention(C.byref(a), None))
    rows = list(range(0, 900, 37)) + [63, 64, 575, 576, 639, 640, 899]
    want = plain_mixed(q[rows], k[0], v[0], [pos[r] for r in rows], win, 0.25, temp, talk)
    assert rel(out.reshape(900, H, dv)[rows], want) < 2e-2


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("shape", [(4, 2, 16, 8), (3, 1, 10, 6), (4, 2, 64, 64)])
def test_temperatures_without_a_mix(S, shape, kind):
    """the row, group and tile kernels of plain softmax attention multiply the scores of a head by its own number"""
    H, G, d, dv = shape
    code, g, PR, n = code_of(S, kind), gen(d), 64, 130
    k, v = {0: rounded(torch.randn(n, G, d, generator=g), kind)}, {0: rounded(torch.randn(n, G, dv, generator=g), kind)}
    q = rounded(torch.randn(100, H, d, generator=g), kind)
    temp = torch.linspace(0.25, 3.0, H, dtype=torch.float64)
    (kp, vp), table, max_pages = paged(S, code, [k, v], PR, 2)
    pos = list(range(30, 130))
    for sel, longest in ((list(range(100)), 100), ([99], 1)):
        out = empty(len(sel), H * dv)
        a = S.PagedAttentionArgs(dev(q[sel].reshape(len(sel), -1), tdt(S, code)).data_ptr(), out.data_ptr(), kp.data_ptr(), vp.data_ptr(), table.data_ptr(),
                                 max_pages, PR, ints([0] * len(sel)).data_ptr(), ints([pos[i] for i in sel]).data_ptr(), len(sel), H, G, d, dv, 0.3, 0.0, 0.0,
                                 code, longest, n, None, 0, 0, 1, 1, 0, 0, None, f32(temp).data_ptr(), None)
        sync_ok(S.lib().b200_paged_attention(C.byref(a), None))
        want = plain_mixed(q[sel], k[0], v[0], [pos[i] for i in sel], 0, 0.3, temp, None)
        assert rel(out.reshape(len(sel), H, dv), want) < (2e-2 if kind == "bf16" else 2e-5)


# ---------------------------------------------------------------------------------------------------------------
SSD_SHAPES = [  # heads, groups, vdim, state
    (4, 2, 24, 20),
    (3, 1, 1, 1),
    (2, 2, 7, 5),
    (4, 1, 64, 128),
    (2, 1, 100, 48),
    (6, 3, 33, 200),
    (1, 1, 130, 256),
]


@pytest.mark.parametrize("chunked", [0, 1])
@pytest.mark.parametrize("shape", SSD_SHAPES)
def test_state_space_recurrence(S, shape, chunked):
    """three sequences over stale slot states: their first portions (200, 3 and 70 tokens) in one call, single tokens of all three
    in the next, then two more portions (150 and 2 tokens) beside a token; step sizes from tiny to large enough to forget
    everything at once"""
    H, G, P, N = shape
    g = gen(sum(shape))
    parts = [[200, 1, 150], [3, 1, 2], [70, 1, 1]]
    lens = [sum(p) for p in parts]
    ch = H * P + 2 * G * N
    u = [torch.randn(n, ch + 3, generator=g, dtype=torch.float32).double() for n in lens]          # a leading dimension of its own
    raw = [(torch.randn(n, H + 1, generator=g, dtype=torch.float32) * 3 - 1).double() for n in lens]
    bias, A_log = torch.randn(H, generator=g).double(), (torch.randn(H, generator=g) * 1.5).float().double()
    D = torch.randn(H, generator=g).double()
    want = []
    for uu, r in zip(u, raw):
        n = len(uu)
        x, B, Cc = uu[:, :H * P].reshape(n, H, P), uu[:, H * P:H * P + G * N].reshape(n, G, N), uu[:, H * P + G * N:ch].reshape(n, G, N)
        want.append(O.ssd(x, B, Cc, torch.nn.functional.softplus(r[:, :H] + bias.float().double(), threshold=1e9), A_log, D).reshape(n, H * P))
    slots = [2, 0, 3]
    state = empty(4, H * N * P, fill=1e3)                                   # stale: a sequence that starts at 0 must not read it
    A = f32(-torch.exp(A_log))
    at, got = [0, 0, 0], [[], [], []]
    for call in range(3):
        cnt = [p[call] for p in parts]
        uu = torch.cat([u[i][at[i]:at[i] + cnt[i]] for i in range(3)])
        rr = torch.cat([raw[i][at[i]:at[i] + cnt[i]] for i in range(3)])
        T = len(uu)
        out = empty(T, H * P, fill=float("nan"))
        a = S.SsdScanArgs()
        a.u, a.ld_u, a.x_off, a.b_off, a.c_off = f32(uu).data_ptr(), ch + 3, 0, H * P, H * P + G * N
        a.dt_raw, a.ld_dt, a.dt_bias, a.A, a.D = f32(rr).data_ptr(), H + 1, f32(bias).data_ptr(), A.data_ptr(), f32(D).data_ptr()
        a.state, a.out = state.data_ptr(), out.data_ptr()
        a.ent_row, a.ent_len = ints([0, cnt[0], cnt[0] + cnt[1]]).data_ptr(), ints(cnt).data_ptr()
        a.slot = ints(sum([[slots[i]] * cnt[i] for i in range(3)], [])).data_ptr()
        a.pos = ints(sum([list(range(at[i], at[i] + cnt[i])) for i in range(3)], [])).data_ptr()
        a.n_entries, a.n_tokens, a.heads, a.groups, a.vdim, a.n_state = 3, T, H, G, P, N
        a.longest_entry, a.chunked = max(cnt), chunked
        need = S.lib().b200_ssd_scan_workspace_bytes(T, 3, H, G, P, N)
        ws = torch.full((max(need, 16),), 255, dtype=torch.uint8, device="cuda")
        _alive.append(ws)
        a.workspace, a.workspace_bytes = ws.data_ptr(), need
        sync_ok(S.lib().b200_ssd_scan(C.byref(a), None))
        o = 0
        for i in range(3):
            got[i].append(out[o:o + cnt[i]].clone())
            o += cnt[i]
            at[i] += cnt[i]
    for i in range(3):
        assert rel(torch.cat(got[i]), want[i]) < (3e-3 if chunked else 5e-6), i
    assert float(state[1].min()) == 1e3                                     # the slot nobody used


def test_recurrence_with_step_sizes_that_add_up_to_thousands(S):
    """decay exponents whose running sum inside a chunk reaches thousands: neighbours still have to decay by exactly their own"""
    H, P, N, T = 1, 8, 16, 256
    g = gen(4)
    u = torch.randn(T, P + 2 * N, generator=g).double()
    raw = torch.where(torch.arange(T)[:, None] % 7 == 3, torch.tensor(60.0), torch.tensor(-9.0)).double()
    A_log = torch.tensor([2.5], dtype=torch.float64)
    want = O.ssd(u[:, :P].reshape(T, 1, P), u[:, P:P + N].reshape(T, 1, N), u[:, P + N:].reshape(T, 1, N),
                 torch.nn.functional.softplus(raw, threshold=1e9), A_log, torch.zeros(1, dtype=torch.float64)).reshape(T, P)
    for chunked, tol in ((0, 5e-6), (1, 2e-3)):
        out, state = empty(T, P), empty(1, N * P)
        need = S.lib().b200_ssd_scan_workspace_bytes(T, 1, 1, 1, P, N)
        ws = empty(need // 4 + 4)
        a = S.SsdScanArgs(f32(u).data_ptr(), P + 2 * N, 0, P, P + N, f32(raw).data_ptr(), 1, f32(torch.zeros(1)).data_ptr(), f32(-torch.exp(A_log)).data_ptr(),
                          f32(torch.zeros(1)).data_ptr(), state.data_ptr(), out.data_ptr(), ints([0]).data_ptr(), ints([T]).data_ptr(), ints([0] * T).data_ptr(),
                          ints(list(range(T))).data_ptr(), 1, T, 1, 1, P, N, T, chunked, ws.data_ptr(), need)
        sync_ok(S.lib().b200_ssd_scan(C.byref(a), None))
        # row by row: small rows follow a step that wiped the state (a few are small because C . B cancels: tf32 products there)
        e = (out.double().cpu() - want).abs().amax(1) / want.abs().amax(1)
        assert float(e.quantile(0.97)) < tol * 10 and rel(out, want) < tol, chunked


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("n,parts", [(1, 1), (12, 3), (30, 2), (384, 2), (4096, 1), (4096, 8), (5000, 4), (9000, 1)])
def test_gated_norm_in_parts(S, n, parts, kind):
    code, g, T = code_of(S, kind), gen(n), 5
    y, z, w = torch.randn(T, n, generator=g), torch.randn(T, n + 4, generator=g), 1 + torch.randn(n, generator=g) * 0.2
    out = empty(T, n, dtype=tdt(S, code))
    sync_ok(S.lib().b200_gated_group_rms(f32(y).data_ptr(), f32(z).data_ptr(), n + 4, f32(w).data_ptr(), out.data_ptr(), T, n, parts, 1e-5, code, None))
    want = O.gated_group_norm(y.double(), z[:, :n].double(), w.double(), parts, 1e-5)
    assert rel(out.float(), want) < (1e-2 if kind == "bf16" else 2e-6)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width", [1, 7, 256, 300, 5504])
def test_activation_of_normed_powers(S, width, kind):
    code, g, T = code_of(S, kind), gen(width), 4
    z, c4 = torch.randn(T, width, generator=g) * torch.tensor([0.01, 1.0, 5.0, 40.0])[:, None], torch.tensor([0.7, -0.4, 0.3, 0.2])
    out = empty(T, width, dtype=tdt(S, code))
    sync_ok(S.lib().b200_poly_norm(f32(z).data_ptr(), f32(c4).data_ptr(), 1e-6, out.data_ptr(), T, width, code, None))
    want = O.poly_norm(z.double(), c4.float().double().tolist(), 1e-6)
    for t in range(T):
        assert rel(out[t].float(), want[t]) < (1e-2 if kind == "bf16" else 3e-6), t


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("width", [1, 5, 48, 300, 2048, 5000, 9000])
def test_parallel_residual_update(S, width, kind):
    """all addends with both norms and experts, then one plain addend without a following norm"""
    code, g, T, top = code_of(S, kind), gen(width), 6, 3
    x, y1, y2, y3 = (torch.randn(T, width, generator=g) * s for s in (1.0, 3.0, 0.1, 1.0))
    w1, w2, lw, lb = (1 + torch.randn(width, generator=g) * 0.2 for _ in range(4))
    eo = torch.randn(T * top, width, generator=g)
    dest = torch.randperm(T * top, generator=g).view(T, top)
    wt = torch.rand(T, top, generator=g)
    dx, out = f32(x), empty(T, width, dtype=tdt(S, code))
    a = S.ParallelResidualArgs()
    a.x, a.mult, a.y1, a.w1, a.s1 = dx.data_ptr(), 0.7, f32(y1).data_ptr(), f32(w1).data_ptr(), 0.5
    a.y2, a.w2, a.s2, a.y3 = f32(y2).data_ptr(), f32(w2).data_ptr(), 0.25, f32(y3).data_ptr()
    a.expert_out, a.dest, a.weight, a.top = f32(eo).data_ptr(), ints(dest).data_ptr(), f32(wt).data_ptr(), top
    a.ln_w, a.ln_b, a.eps, a.out, a.out_dtype, a.n_rows, a.width = f32(lw).data_ptr(), f32(lb).data_ptr(), 1e-5, out.data_ptr(), code, T, width
    sync_ok(S.lib().b200_parallel_residual(C.byref(a), None))
    ex = (eo.double()[dest.reshape(-1)].view(T, top, width) * wt.double()[:, :, None]).sum(1)
    m = float(torch.tensor(0.7))
    want = x.double() + m * (0.5 * O.rms_norm(y1.double(), w1.double(), 1e-5) + 0.25 * O.rms_norm(y2.double(), w2.double(), 1e-5) + y3.double() + ex)
    assert rel(dx, want) < 2e-6
    if width > 1:
        assert rel(out.float(), O.layer_norm(want, lw.double(), 1e-5) + lb.double()) < (1e-2 if kind == "bf16" else 1e-5)
    b = S.ParallelResidualArgs()
    b.x, b.mult, b.y1, b.s1, b.eps, b.n_rows, b.width = dx.data_ptr(), 2.0, f32(y1).data_ptr(), 1.0, 1e-5, T, width
    sync_ok(S.lib().b200_parallel_residual(C.byref(b), None))
    assert rel(dx, want + 2 * y1.double()) < 2e-6


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("experts,top,count,keep", [(15, 4, 5, 3), (8, 2, 1, 1), (1, 1, 1, 1), (64, 6, 8, 2), (30, 5, 5, 1), (40, 16, 40, 20), (6, 6, 2, 2)])
def test_router_with_groups(S, experts, top, count, keep, kind):
    code, g, T, D = code_of(S, kind), gen(experts + top), 50, 40
    h = rounded(torch.randn(T, D, generator=g), kind)
    wr = torch.randn(experts, D, generator=g).double() * 0.5
    if count > 1:
        wr[experts // count - 1] *= 4.0            # a group with one outstanding expert among weak ones
    chosen, weight = empty(T, top, dtype=torch.int32), empty(T, top)
    sync_ok(S.lib().b200_moe_route_groups(dev(h, tdt(S, code)).data_ptr(), code, f32(wr).data_ptr(), T, D, experts, top, count, keep, chosen.data_ptr(),
                                          weight.data_ptr(), None))
    wc, ww = O.route(h @ wr.float().double().T, dict(count=count, keep=keep), top)
    gc, gw = chosen.cpu().long(), weight.cpu().double()
    for t in range(T):
        assert sorted(gc[t].tolist()) == sorted(wc[t].tolist()), t
        mine = dict(zip(gc[t].tolist(), gw[t].tolist()))
        for e, w in zip(wc[t].tolist(), ww[t].tolist()):
            assert abs(mine[e] - w) < 1e-5, (t, e)
    bad = S.lib().b200_moe_route_groups(dev(h, tdt(S, code)).data_ptr(), code, f32(wr).data_ptr(), T, D, experts, top, experts + 1, 1, chosen.data_ptr(),
                                        weight.data_ptr(), None)
    assert bad != 0


def test_equal_scores_take_the_lower_index(S):
    h, wr = torch.zeros(3, 8), torch.zeros(12, 8)
    chosen, weight = empty(3, 4, dtype=torch.int32), empty(3, 4)
    sync_ok(S.lib().b200_moe_route_groups(f32(h).data_ptr(), S.F32, f32(wr).data_ptr(), 3, 8, 12, 4, 3, 2, chosen.data_ptr(), weight.data_ptr(), None))
    assert chosen.cpu().tolist() == [[0, 1, 2, 3]] * 3 and torch.allclose(weight.cpu(), torch.full((3, 4), 0.25))


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("Q,R,dr", [(1, 1, 2), (12, 20, 6), (96, 72, 0), (300, 512, 64)])
def test_low_rank_norms_and_the_rotated_key_part(S, Q, R, dr, kind):
    code, g, PR, T, start = code_of(S, kind), gen(Q), 64, 40, 50
    ld, kv = Q + R + dr + 5, Q + 2
    raw = torch.randn(T, ld, generator=g)
    qn, kn = 1 + torch.randn(Q, generator=g) * 0.2, 1 + torch.randn(R, generator=g) * 0.2
    pos = list(range(start, start + T))
    f = [500.0 ** (-2.0 * i / dr) for i in range(dr // 2)] if dr else []
    ang = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
    table = ints([[0, 0], [3, 1]])
    pool, q_out = empty(4 * PR, R + dr, dtype=tdt(S, code), fill=7.0), empty(T, Q, dtype=tdt(S, code))
    a = S.LatentNormsArgs()
    a.raw, a.ld_raw, a.q_off, a.kv_off, a.q_norm, a.q_rank, a.q_out = f32(raw).data_ptr(), ld, 0, kv, f32(qn).data_ptr(), Q, q_out.data_ptr()
    a.kv_norm, a.eps, a.pool, a.pages, a.max_pages, a.page_rows = f32(kn).data_ptr(), 1e-5, pool.data_ptr(), table.data_ptr(), 2, PR
    a.slot, a.pos, a.n_tokens, a.rank, a.extra = ints([1] * T).data_ptr(), ints(pos).data_ptr(), T, R, dr
    a.cos, a.sin, a.rot_layout, a.dtype = f32(torch.cos(ang)).data_ptr(), f32(torch.sin(ang)).data_ptr(), S.ROPE_HALF, code
    sync_ok(S.lib().b200_latent_norms(C.byref(a), None))
    tol = 1e-2 if kind == "bf16" else 3e-6
    assert rel(q_out.float(), O.rms_norm(raw[:, :Q].double(), qn.double(), 1e-5)) < tol
    full = torch.zeros(start + T, 1, dr, dtype=torch.float64)
    full[start:, 0] = raw[:, kv + R:kv + R + dr].double()
    want = torch.cat([O.rms_norm(raw[:, kv:kv + R].double(), kn.double(), 1e-5), O.turn_half(full, dict(base=500.0, dims=dr))[start:, 0]], 1)
    rows = [(3 if p < PR else 1) * PR + p % PR for p in pos]
    assert rel(pool[rows].float(), want) < tol
    untouched = sorted(set(range(4 * PR)) - set(rows))
    assert float((pool[untouched].float() - 7.0).abs().max()) == 0.0
    before = pool.clone()
    a.pool = None                                  # a layer that reads another layer's rows only norms its queries
    sync_ok(S.lib().b200_latent_norms(C.byref(a), None))
    assert torch.equal(pool, before)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_layer_norm_without_bias(S, kind):
    code, g = code_of(S, kind), gen(3)
    x, w = torch.randn(9, 50, generator=g) + 3.0, 1 + torch.randn(50, generator=g) * 0.2
    out = empty(4, 50, dtype=tdt(S, code))
    rows = [8, 0, 3, 3]
    sync_ok(S.lib().b200_layernorm_pair(f32(x).data_ptr(), ints(rows).data_ptr(), 4, 50, 1e-5, f32(w).data_ptr(), None, out.data_ptr(), None, None, None, code, None))
    assert rel(out.float(), O.layer_norm(x.double(), w.double(), 1e-5)[rows]) < (1e-2 if kind == "bf16" else 3e-6)
