"""Plain, slow statement of the Filipel decoder, one function per mechanism (torch on the CPU, float64).

Shares no code with the product path: the tests build small random models, run them through the library and compare
with these functions. Every function sees a WHOLE sequence from position 0; nothing is cached.

Design: parallel layers, x <- x + m (mixer(N x) + ff(N x)) with one layer norm (a weight, no bias) read by both sublayers
and one multiplier m. Two mixers: "latent_attention" (queries through a normed low-rank row, keys and values expanded from a
cached normed latent row plus one rotary key part shared by the heads, an element-wise sigmoid output gate; a layer may read
the latent rows of an earlier layer) and "parallel" (windowed grouped-query attention whose softmax weights are mixed across
the heads before they meet the values, beside a state-space recurrence with one decay per head; each output is RMS-normed,
the mixer is half their sum). Feed-forward: none, a dense one with a polynomial activation of normed powers, or a routed
mixture of gated experts whose choice is limited to the best groups of experts.

A model is (config dict as in config.json, dict name -> tensor).
"""
import math

import torch

DT = torch.float64


def silu(z):
    return z * torch.sigmoid(z)


def unit_rms(y, eps):
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def rms_norm(y, w, eps):
    return unit_rms(y, eps) * w


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def turn_half(x, rot):
    """x [T, heads, n], token t at position t: dimensions m and m + dims/2 (m < dims/2) turned by t * base^(-2m/dims)"""
    if not rot or not rot.get("dims"):
        return x
    P = rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2.0 * m / rot["dims"]) for m in range(P)], dtype=DT)
    ang = torch.arange(x.shape[0], dtype=DT)[:, None, None] * f
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :P], x[..., P:2 * P]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * P:]], -1)


def visible(T, size):
    """[T, T] bool: key j seen by position i (causal; with a window size only the last `size` positions, i's own included)"""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < size) if size else back >= 0


def softmax_weights(q, k, group, scale, temp, ok):
    """[H, T, T] softmax weights; q [T, H, d], k [T, G, d], head h against key head h // group; temp [H]"""
    s = torch.stack([q[:, h] @ k[:, h // group].T * scale * temp[h] for h in range(q.shape[1])])
    return torch.softmax(s.masked_fill(~ok, float("-inf")), -1)


def latent_rows(h, mx, W, pre, eps):
    """what a latent layer caches: the normed latent and the rotated key part"""
    R = mx["kv_rank"]
    raw = h @ W[pre + "dkv"].T
    return rms_norm(raw[:, :R], W[pre + "dkv.norm"], eps), turn_half(raw[:, None, R:], mx.get("rot"))[:, 0]


def latent_attention(h, rows, mx, W, pre, eps):
    T, H, d, dr, dv = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    c, kr = rows
    q = (rms_norm(h @ W[pre + "dq"].T, W[pre + "dq.norm"], eps) @ W[pre + "uq"].T).view(T, H, d + dr)
    qr = turn_half(q[..., d:], mx.get("rot"))
    kn, v = (c @ W[pre + "uk"].T).view(T, H, d), (c @ W[pre + "uv"].T).view(T, H, dv)
    ok = visible(T, 0)
    out = []
    for a in range(H):
        s = (q[:, a, :d] @ kn[:, a].T + qr[:, a] @ kr.T) * mx["scale"]
        out.append(torch.softmax(s.masked_fill(~ok, float("-inf")), -1) @ v[:, a])
    return (torch.cat(out, -1) * torch.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def mixed_attention(q, k, v, scale, temp, talk, size):
    """windowed softmax weights, w_h <- sum_g talk[h, g] w_g, then the values of h's own key head. Returns [T, H, dv]"""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    p = softmax_weights(q, k, H // G, scale, temp, visible(T, size))
    p = torch.einsum("hg,gij->hij", talk, p)
    return torch.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def talking_attention(h, mx, W, pre):
    T, H, G, d, dv = h.shape[0], mx["heads"], mx.get("kv_heads", mx["heads"]), mx["dim"], mx["vdim"]
    q, k, v = ((h @ W[pre + n].T).view(T, a, b) for n, a, b in (("q", H, d), ("k", G, d), ("v", G, dv)))
    q, k = turn_half(q, mx.get("rot")), turn_half(k, mx.get("rot"))
    o = mixed_attention(q, k, v, mx["scale"], W[pre + "temp"], W[pre + "talk"], (mx.get("mask") or {}).get("size", 0))
    return (o.reshape(T, H * dv) * torch.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def causal_conv_silu(u, w, b):
    """u [T, C], w [C, taps] (last column: the current token), zeros before the start"""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=DT), u])
    return silu(sum(padded[j: j + u.shape[0]] * w[:, j] for j in range(taps)) + b)


def ssd(x, B, C, dt, A_log, D):
    """S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T; y_t = S_t^T C_t + D x_t. x [T, H, P], B, C [T, G, N], dt [T, H]"""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=DT)
    grp = torch.arange(H) // (H // G)
    y = []
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][grp][:, :, None] * x[t][:, None, :]
        y.append((S * C[t][grp][:, :, None]).sum(1) + D[:, None] * x[t])
    return torch.stack(y)


def gated_group_norm(y, z, w, groups, eps):
    """y silu(z), each of `groups` equal parts divided by its own root mean square, times w"""
    v = (y * silu(z)).view(y.shape[0], groups, -1)
    return unit_rms(v, eps).reshape(y.shape) * w


def state_space(h, mx, W, pre, eps):
    T, H, P, N, G = h.shape[0], mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * P
    z, u, dt = torch.split(h @ W[pre + "in"].T, [inner, inner + 2 * G * N, H], -1)
    u = causal_conv_silu(u, W[pre + "conv"], W[pre + "conv.b"])
    x, B, C = torch.split(u, [inner, G * N, G * N], -1)
    y = ssd(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), torch.nn.functional.softplus(dt + W[pre + "dt_bias"], threshold=1e9),
            W[pre + "A_log"], W[pre + "D"])
    return gated_group_norm(y.reshape(T, inner), z, W[pre + "norm"], mx["norm_groups"], eps) @ W[pre + "o"].T


def parallel_mixer(h, mx, W, pre, eps):
    left = talking_attention(h, mx["left"], W, pre + "left.")
    right = state_space(h, mx["right"], W, pre + "right.", eps)
    return 0.5 * (rms_norm(left, W[pre + "left.out"], eps) + rms_norm(right, W[pre + "right.out"], eps))


def poly_norm(z, abce, eps):
    a, b, c, e = abce
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def route(z, groups, top):
    """(chosen [T, top], weight [T, top]) from router logits: softmax over all experts, the best `keep` of `count` groups by
    their largest score, the `top` largest scores inside them, weights divided by their sum"""
    s = torch.softmax(z, -1)
    count, keep = (groups["count"], groups["keep"]) if groups else (1, 1)
    best = s.view(z.shape[0], count, -1).amax(-1).topk(keep, -1).indices
    allowed = torch.zeros(z.shape[0], count, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(z.shape[1] // count, 1)
    chosen = s.masked_fill(~allowed, -1.0).topk(top, -1).indices
    w = s.gather(1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20)


def feed_forward(h, ml, W, pre, eps):
    if ml["kind"] == "dense":
        return poly_norm(h @ W[pre + "up"].T, W[pre + "act"], eps) @ W[pre + "down"].T
    ro = ml["router"]
    chosen, wt = route(h @ W[pre + "router"].T, ro.get("groups"), ro["top"])
    out = torch.zeros_like(h)
    for e in range(ro["experts"]):
        t, k = (chosen == e).nonzero(as_tuple=True)
        if len(t):
            p = pre + "e%d." % e
            y = (silu(h[t] @ W[p + "gate"].T) * (h[t] @ W[p + "up"].T)) @ W[p + "down"].T
            out[t] += wt[t, k][:, None] * y
    return out


def forward(cfg, W, tokens, keep_layers=False):
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    kept, cached = [], {}
    for i, lj in enumerate(cfg["layers"]):
        pre, mx = "l%d." % i, lj["mixer"]
        h = layer_norm(x, W[pre + "norm1"], eps)
        if lj["type"] == "latent_attention":
            if mx.get("kv_from") is None:
                cached[i] = latent_rows(h, mx, W, pre + "mix.", eps)
            y = latent_attention(h, cached[i if mx.get("kv_from") is None else mx["kv_from"]], mx, W, pre + "mix.", eps)
        else:
            y = parallel_mixer(h, mx, W, pre + "mix.", eps)
        if lj.get("mlp"):
            y = y + feed_forward(h, lj["mlp"], W, pre + "mlp.", eps)
        x = x + m * y
        if keep_layers:
            kept.append(x.clone())
    logits = layer_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


class Oracle:
    def __init__(self, cfg, w):
        self.cfg, self.w = cfg, w

    def forward(self, tokens, return_layers=False):
        return forward(self.cfg, self.w, tokens, keep_layers=return_layers)


# ---------------------------------------------------------------------------------------------------------------
# small random models for the tests (weights rounded to bfloat16, as a checkpoint stores them)
# ---------------------------------------------------------------------------------------------------------------
def random_model(seed, width, vocab, layers, mult=0.5, eps=1e-5):
    """layers: dicts with type 'latent_attention' (heads, dim, rot_dim, vdim, q_rank, kv_rank, optionally base, scale, kv_from)
    | 'parallel' (left = dict(heads, kv_heads, dim, vdim, optionally rot_dims, base, scale, window, sharp), right = dict(heads,
    vdim, state, groups, conv, norm_groups)); ff = None | int (dense) | (ff, experts, top, groups, keep)."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=None):
        return torch.randn(*shape, generator=g, dtype=torch.float32) * (s if s is not None else 1.0 / math.sqrt(shape[-1]))

    cfg = dict(architecture="Filipel", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, layers=[])
    w = {"embed": rnd(vocab, width, s=1.0), "head": rnd(vocab, width), "final.norm": 1 + rnd(width, s=0.1)}
    for i, sp in enumerate(layers):
        pre = "l%d." % i
        mp = pre + "mix."
        w[pre + "norm1"] = 1 + rnd(width, s=0.1)
        if sp["type"] == "latent_attention":
            H, d, dr, dv, Q, R = sp["heads"], sp["dim"], sp["rot_dim"], sp["vdim"], sp["q_rank"], sp["kv_rank"]
            mx = dict(heads=H, dim=d, rot_dim=dr, vdim=dv, q_rank=Q, kv_rank=R, scale=sp.get("scale", 1.0 / math.sqrt(d + dr)),
                      rot=dict(base=sp.get("base", 10000.0), dims=dr))
            w[mp + "dq"], w[mp + "dq.norm"], w[mp + "uq"] = rnd(Q, width), 1 + rnd(Q, s=0.2), rnd(H * (d + dr), Q, s=2.0 / math.sqrt(Q))
            if sp.get("kv_from") is not None:
                mx["kv_from"] = sp["kv_from"]
            else:
                w[mp + "dkv"], w[mp + "dkv.norm"] = rnd(R + dr, width), 1 + rnd(R, s=0.2)
            w[mp + "uk"], w[mp + "uv"] = rnd(H * d, R, s=2.0 / math.sqrt(R)), rnd(H * dv, R)
            w[mp + "g"], w[mp + "o"] = rnd(H * dv, width), rnd(width, H * dv)
        else:
            a, b = sp["left"], sp["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            left = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=a.get("scale", 1.0 / math.sqrt(d)))
            if a.get("rot_dims", d):
                left["rot"] = dict(base=a.get("base", 10000.0), dims=a.get("rot_dims", d))
            if a.get("window"):
                left["mask"] = dict(size=a["window"])
            lp, rp = mp + "left.", mp + "right."
            sharp = a.get("sharp", 1.5)
            w[lp + "q"], w[lp + "k"], w[lp + "v"] = rnd(H * d, width, s=sharp / math.sqrt(width)), rnd(G * d, width, s=sharp / math.sqrt(width)), rnd(G * dv, width)
            w[lp + "temp"] = 1 + rnd(H, s=0.3)
            w[lp + "talk"] = 0.7 * torch.eye(H) + rnd(H, H, s=0.6 / math.sqrt(H))
            w[lp + "g"], w[lp + "o"], w[lp + "out"] = rnd(H * dv, width), rnd(width, H * dv), 1 + rnd(width, s=0.2)
            Hs, P, N, Gs, taps = b["heads"], b["vdim"], b["state"], b["groups"], b["conv"]
            right = dict(heads=Hs, vdim=P, state=N, groups=Gs, conv=taps, norm_groups=b["norm_groups"])
            ch = Hs * P + 2 * Gs * N
            w[rp + "in"] = rnd(Hs * P + ch + Hs, width)
            w[rp + "conv"], w[rp + "conv.b"] = rnd(ch, taps, s=0.8), rnd(ch, s=0.2)
            w[rp + "dt_bias"], w[rp + "A_log"], w[rp + "D"] = rnd(Hs, s=1.0) - 2.0, rnd(Hs, s=0.7), 1 + rnd(Hs, s=0.3)
            w[rp + "norm"], w[rp + "o"], w[rp + "out"] = 1 + rnd(Hs * P, s=0.2), rnd(width, Hs * P), 1 + rnd(width, s=0.2)
            mx = dict(left=left, right=right)
        ff = sp.get("ff")
        if ff is None:
            ml = None
        elif isinstance(ff, int):
            ml = dict(kind="dense", ff=ff)
            w[pre + "mlp.up"], w[pre + "mlp.down"] = rnd(ff, width), rnd(width, ff)
            w[pre + "mlp.act"] = torch.tensor([0.6, 0.4, 0.3, -0.2]) + rnd(4, s=0.1)
        else:
            f, E, top, gc, keep = ff
            ml = dict(kind="moe", expert=dict(ff=f), router=dict(experts=E, top=top))
            if gc:
                ml["router"]["groups"] = dict(count=gc, keep=keep)
            w[pre + "mlp.router"] = rnd(E, width, s=2.0 / math.sqrt(width))
            for e in range(E):
                p = pre + "mlp.e%d." % e
                w[p + "gate"], w[p + "up"], w[p + "down"] = rnd(f, width), rnd(f, width), rnd(width, f)
        cfg["layers"].append(dict(type=sp["type"], mixer=mx, mlp=ml))
    return cfg, {k: v.to(torch.bfloat16).to(DT) for k, v in w.items()}


def write_model(folder, cfg, w):
    """config.json + model.safetensors with every tensor as bfloat16"""
    import json
    import os
    import struct

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, off = {}, [], 0
    for name, t in w.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        header[name] = dict(dtype="BF16", shape=list(t.shape), data_offsets=[off, off + len(raw)])
        blobs.append(raw)
        off += len(raw)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)))
        f.write(hj)
        for b in blobs:
            f.write(b)
