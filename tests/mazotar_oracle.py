"""Plain, slow statement of the Mazotar decoder, one function per mechanism (torch on the CPU, float64).

Shares no code with the product path: the tests build small random models, run them through the library and compare
with these functions. Every function sees a WHOLE sequence from position 0; nothing is cached.

Design: a token embedding (scaled) plus fixed sinusoids of the position, copied into `streams` parallel residual streams.
Every sublayer reads one weighted sum of the streams through an RMS norm and writes back into all of them through a small
mixing matrix and an output vector; at the end the streams are summed. Mixers: attention (one RMS norm over the whole query
and the whole key projection, a query temperature that grows with the logarithm of the position, a learned bias per bucket
of the distance, a softmax with a learned sink per head; a layer may read an earlier layer's keys and values) and the matrix
memory of an mLSTM (exponential input gate and sigmoid forget gate, stabilised by a running maximum). Feed-forward: none, a
gated dense one, or a routed mixture whose sigmoid weights multiply the experts' INPUT, beside a shared expert with a sigmoid
gate of its own.

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


def sinusoids(T, width):
    """[T, width]: entries 2i and 2i + 1 are sine and cosine of t / 10000^(2i / width)"""
    out = torch.zeros(T, width, dtype=DT)
    for t in range(T):
        for c in range(width):
            ang = t * 10000.0 ** (-2.0 * (c // 2) / width)
            out[t, c] = math.cos(ang) if c % 2 else math.sin(ang)
    return out


def bucket(n, rows, farthest):
    """row of the distance-bias table for distance n: exact below rows / 2, then logarithmic up to `farthest`"""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(farthest / half) * (rows - half)))


def distance_bias(T, rel, farthest):
    """[H, T, T] (query i, key j <= i; zero elsewhere)"""
    rows = rel.shape[0]
    of = torch.tensor([bucket(n, rows, farthest) for n in range(T)])
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :])
    return torch.where(back[None] >= 0, rel[of[back.clamp_min(0)]].permute(2, 0, 1), torch.zeros((), dtype=DT))


def temperature(T, coef, every):
    return torch.tensor([1 + coef * math.log((t + 1) // every + 1) for t in range(T)], dtype=DT)


def sink_softmax(s, sink):
    """softmax over the last axis of s [H, T, n] whose denominator also holds exp(sink[h])"""
    m = torch.maximum(s.amax(-1), sink[:, None])
    e = torch.exp(s - m[..., None])
    return e / (e.sum(-1) + torch.exp(sink[:, None] - m))[..., None]


def attend(q, k, v, scale, bias, sink):
    """q [T, H, d], k [n = T, G, d], v [n, G, dv]; bias [H, T, T]"""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = torch.stack([q[:, h] @ k[:, h // (H // G)].T for h in range(H)]) * scale + bias
    p = sink_softmax(s.masked_fill(back < 0, float("-inf")), sink)
    return torch.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def keys_and_values(h, mx, W, pre, eps):
    """what an attention layer caches: normed keys [T, G, d] and values [T, G, dv]"""
    T, G = h.shape[0], mx["kv_heads"]
    k = rms_norm(h @ W[pre + "k"].T, W[pre + "k.norm"], eps)
    return k.view(T, G, mx["dim"]), (h @ W[pre + "v"].T).view(T, G, mx["vdim"])


def attention(h, kv, mx, W, pre, eps):
    T, H = h.shape[0], mx["heads"]
    q = rms_norm(h @ W[pre + "q"].T, W[pre + "q.norm"], eps).view(T, H, mx["dim"])
    qt = mx.get("q_temp")
    if qt:
        q = q * temperature(T, qt["coef"], qt["every"])[:, None, None]
    o = attend(q, *kv, mx["scale"], distance_bias(T, W[pre + "rel"], mx["bias_max"]), W[pre + "sink"])
    return o.reshape(T, -1) @ W[pre + "o"].T


def mlstm_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, p], log gates i, f [T, H]: the stabilised recurrence, token by token. [T, H, p]"""
    T, H, d = q.shape
    S, n, m = torch.zeros(H, d, v.shape[2], dtype=DT), torch.zeros(H, d, dtype=DT), torch.zeros(H, dtype=DT)
    out = []
    for t in range(T):
        m2 = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m2), torch.exp(i[t] - m2)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = m2
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][:, :, None]).sum(1) / den[:, None])
    return torch.stack(out)


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm(h, mx, W, pre, eps):
    T, H, d, p = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q, k, v = ((h @ W[pre + n].T).view(T, H, -1) for n in "qkv")
    i = capped(h @ W[pre + "i"].T + W[pre + "i.b"], mx["gate_cap"])
    f = torch.nn.functional.logsigmoid(capped(h @ W[pre + "f"].T + W[pre + "f.b"], mx["gate_cap"]))
    o = unit_rms(mlstm_memory(q * d ** -0.5, k, v, i, f), eps).reshape(T, H * p)
    return (o * W[pre + "norm"] * torch.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def gated_unit(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, top):
    """(chosen [T, top], weight [T, top]) from router logits: the largest sigmoids, as they are"""
    s = torch.sigmoid(z)
    chosen = z.topk(top, -1).indices
    return chosen, s.gather(1, chosen)


def feed_forward(h, ml, W, pre):
    if ml["kind"] == "dense":
        return gated_unit(h, W, pre)
    chosen, wt = route(h @ W[pre + "router"].T, ml["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(ml["router"]["experts"]):
        t, k = (chosen == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += gated_unit(wt[t, k][:, None] * h[t], W, pre + "e%d." % e)
    if ml.get("shared"):
        out = out + torch.sigmoid(h @ W[pre + "shared.sg"].T) * gated_unit(h, W, pre + "shared.")
    return out


def hyper(x, W, pre, norm, eps, sublayer):
    """x [s, T, D] -> the streams after one sublayer"""
    u = torch.einsum("s,std->td", W[pre + "in"], x)
    y = sublayer(rms_norm(u, norm, eps))
    return torch.einsum("sr,std->rtd", W[pre + "mix"], x) + W[pre + "out"][:, None, None] * y


def forward(cfg, W, tokens, keep_layers=False):
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"] + sinusoids(len(tokens), cfg["width"])
    x = x.repeat(cfg["streams"], 1, 1)
    kept, cached = [], {}
    for i, lj in enumerate(cfg["layers"]):
        pre, mx = "l%d." % i, lj["mixer"]

        def mixer(h):
            if lj["type"] == "mlstm":
                return mlstm(h, mx, W, pre + "mix.", eps)
            j = mx.get("kv_from")
            if j is None:
                cached[i] = keys_and_values(h, mx, W, pre + "mix.", eps)
            return attention(h, cached[i if j is None else j], mx, W, pre + "mix.", eps)
        x = hyper(x, W, pre + "hc1.", W[pre + "norm1"], eps, mixer)
        if lj.get("mlp"):
            x = hyper(x, W, pre + "hc2.", W[pre + "norm2"], eps, lambda h: feed_forward(h, lj["mlp"], W, pre + "mlp."))
        if keep_layers:
            kept.append(x.sum(0))
    logits = rms_norm(x.sum(0), W["final.norm"], eps) @ W["head"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


class Oracle:
    def __init__(self, cfg, w):
        self.cfg, self.w = cfg, w

    def forward(self, tokens, return_layers=False):
        return forward(self.cfg, self.w, tokens, keep_layers=return_layers)


# ---------------------------------------------------------------------------------------------------------------
# small random models for the tests (weights rounded to bfloat16, as a checkpoint stores them)
# ---------------------------------------------------------------------------------------------------------------
def random_model(seed, width, vocab, layers, streams=2, scale=1.5, eps=1e-5):
    """layers: dicts with type 'attention' (heads, kv_heads, dim, vdim, buckets, bias_max, optionally scale, temp = (coef, every) or
    None, kv_from, sharp) | 'mlstm' (heads, dim, vdim, cap); ff = None | int (dense) | (ff, experts, top, shared ff or None)."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=None):
        return torch.randn(*shape, generator=g, dtype=torch.float32) * (s if s is not None else 1.0 / math.sqrt(shape[-1]))

    cfg = dict(architecture="Mazotar", vocab=vocab, width=width, streams=streams, norm=dict(eps=eps), embedding=dict(scale=scale), layers=[])
    w = {"embed": rnd(vocab, width, s=1.0), "head": rnd(vocab, width), "final.norm": 1 + rnd(width, s=0.1)}

    def sublayer(pre, q):
        w[f"{pre}norm{q}"] = 1 + rnd(width, s=0.2)
        w[f"{pre}hc{q}.in"] = 0.6 + rnd(streams, s=0.4)
        w[f"{pre}hc{q}.out"] = 1 + rnd(streams, s=0.5)
        w[f"{pre}hc{q}.mix"] = 0.9 * torch.eye(streams) + rnd(streams, streams, s=0.3)

    for i, sp in enumerate(layers):
        pre = "l%d." % i
        mp = pre + "mix."
        sublayer(pre, 1)
        H, d, dv = sp["heads"], sp["dim"], sp["vdim"]
        if sp["type"] == "mlstm":
            mx = dict(heads=H, dim=d, vdim=dv, gate_cap=sp.get("cap", 10.0))
            for nm, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                w[mp + nm] = rnd(rows, width)
            w[mp + "i"], w[mp + "f"] = rnd(H, width, s=1.5 / math.sqrt(width)), rnd(H, width, s=1.5 / math.sqrt(width))
            w[mp + "i.b"], w[mp + "f.b"], w[mp + "norm"] = rnd(H, s=1.0), 3 + rnd(H, s=1.5), 1 + rnd(H * dv, s=0.2)
        else:
            G = sp["kv_heads"]
            mx = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=sp.get("scale", 1.0 / math.sqrt(d)), bias_max=sp["bias_max"])
            if sp.get("temp"):
                mx["q_temp"] = dict(coef=sp["temp"][0], every=sp["temp"][1])
            w[mp + "q"], w[mp + "q.norm"] = rnd(H * d, width), (1 + rnd(H * d, s=0.4)) * sp.get("sharp", 1.5)
            if sp.get("kv_from") is not None:
                mx["kv_from"] = sp["kv_from"]
            else:
                w[mp + "k"], w[mp + "k.norm"], w[mp + "v"] = rnd(G * d, width), 1 + rnd(G * d, s=0.4), rnd(G * dv, width)
            w[mp + "rel"], w[mp + "sink"] = rnd(sp["buckets"], H, s=1.0), 1 + rnd(H, s=1.0)
        w[mp + "o"] = rnd(width, H * dv)
        ff = sp.get("ff")
        if ff is None:
            cfg["layers"].append(dict(type=sp["type"], mixer=mx, mlp=None))
            continue
        sublayer(pre, 2)
        fp = pre + "mlp."

        def unit(p, f):
            w[p + "gate"], w[p + "up"], w[p + "down"] = rnd(f, width), rnd(f, width), rnd(width, f)
        if isinstance(ff, int):
            ml = dict(kind="dense", ff=ff)
            unit(fp, ff)
        else:
            f, E, top, shared = ff
            ml = dict(kind="moe", expert=dict(ff=f), router=dict(experts=E, top=top))
            w[fp + "router"] = rnd(E, width, s=1.5 / math.sqrt(width))
            for e in range(E):
                unit(fp + "e%d." % e, f)
            if shared:
                ml["shared"] = dict(ff=shared)
                unit(fp + "shared.", shared)
                w[fp + "shared.sg"] = rnd(1, width, s=1.5 / math.sqrt(width))
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
