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
