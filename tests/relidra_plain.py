"""Plain float64 restatement of the Relidra design, one function per mechanism, for the tests. It shares no code with the engine.

A model is (cfg, weights): cfg is the config.json tree, weights maps tensor names to torch tensors. The residual of T tokens of one
sequence at positions 0 .. T-1 is S streams X [S, T, W], all of them embed[token] before the first layer.

  sublayer:    u = sum_s in[s] X[s];  y = f(layer_norm(u));  X'[t] = sum_s mix[s, t] X[s] + out[t] y     (all t from the old X)
  layer:       the mixer's sublayer, then the feed-forward's (absent when "mlp" is null)
  order:       layers start .. stop-1 as one block `times` times with the same weights, each pass over a layer with a state of its own
  layer_norm:  (x - mean) / sqrt(mean((x - mean)^2) + eps) * w
  attention:   q = Wq h + bq, k = Wk h + bk, v = k; q, k = unit_rms(rotate_p(.)) with channel pairs (i, i + dims/2) and frequencies
               base^(-2i/dims) / factor; key j visible to i >= j in the same chunk (equal i // size, j // size); softmax of
               scale * q . k whose denominator also holds exp(sink_h); grouped heads; Wo
  delta:       q, k, v = silu(conv(W h)) (causal, per channel, last tap on the current token); q, k over sqrt(sum of squares + 1e-6), q
               times dim^-1/2; b = sigmoid(Wb h); g = exp(-exp(A_log) softplus(Wa h + dt_bias)); per head
               S <- g S; S <- S + k (b (v - S^T k))^T; o = S^T q;  Wo (unit_rms(o) * norm * silu(Wg h))
  ff:          Wd gelu(Wu h), gelu(z) = z Phi(z)
  readout:     embed . layer_norm(sum_s X[s])
"""
import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def layer_norm(x, w, eps):
    x = x.to(F64)
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w.to(F64)


def unit_rms(x, eps):
    x = x.to(F64)
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_l2(x, eps=UNIT_EPS):
    x = x.to(F64)
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def silu(x):
    return x / (1.0 + torch.exp(-x))


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def gelu_exact(z):
    z = z.to(F64)
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ---- streams ---------------------------------------------------------------------------------------------------------------------------

def streams_read(X, w_in):
    """X [S, T, W], w_in [S] -> what the sublayer's norm reads [T, W]"""
    return torch.einsum("stw,s->tw", X.to(F64), w_in.to(F64))


def streams_write(X, y, w_mix, w_out):
    """new stream t = sum_s mix[s, t] X[s] + out[t] y"""
    return torch.einsum("srw,st->trw", X.to(F64), w_mix.to(F64)) + w_out.to(F64)[:, None, None] * y.to(F64)[None]


# ---- attention -------------------------------------------------------------------------------------------------------------------------

def rot_frequencies(rot):
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    return [base ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate_halves(x, positions, rot):
    """x [T, heads, n]: channel i pairs with channel i + dims/2 (i < dims/2); channels from `dims` on pass unchanged."""
    x = x.to(F64)
    dims = int(rot["dims"])
    half = dims // 2
    ang = torch.as_tensor(positions, dtype=F64)[:, None] * torch.tensor(rot_frequencies(rot), dtype=F64)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    out = x.clone()
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def chunk_mask(pos_q, pos_k, size):
    """seen[i, j]: not in the future and in the same chunk of `size` positions (size 0: one chunk without end)"""
    q, k = torch.as_tensor(pos_q)[:, None], torch.as_tensor(pos_k)[None, :]
    seen = k <= q
    if size:
        seen = seen & (q // size == k // size)
    return seen


def sink_attention(q, k, v, seen, scale, sink):
    """q [Tq, H, d], k [Tk, G, d], v [Tk, G, dv], seen [Tq, Tk] -> [Tq, H, dv]; sink [H] or None"""
    Tq, H = q.shape[0], q.shape[1]
    G = k.shape[1]
    kk, vv = k.to(F64).repeat_interleave(H // G, dim=1), v.to(F64).repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->ihj", q.to(F64), kk) * scale
    s = s.masked_fill(~seen[:, None, :], -math.inf)
    if sink is not None:
        s = torch.cat([s, sink.to(F64)[None, :, None].expand(Tq, H, 1)], dim=2)
    w = torch.softmax(s, dim=2)
    if sink is not None:
        w = w[..., :-1]
    return torch.einsum("ihj,jhv->ihv", w, vv)


def attention_mixer(h, W, p, mc, eps, positions, past=None):
    """past = (k rotated and normed, v, positions) of the tokens before -> (output [T, width], the same with these tokens)"""
    h = h.to(F64)
    T = h.shape[0]
    H, G, d, dv = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
    q = (h @ W[p + "mix.q"].to(F64).T + W[p + "mix.q.b"].to(F64)).reshape(T, H, d)
    k = (h @ W[p + "mix.k"].to(F64).T + W[p + "mix.k.b"].to(F64)).reshape(T, G, d)
    v = k.clone()
    assert dv == d
    if mc.get("rot"):
        q, k = rotate_halves(q, positions, mc["rot"]), rotate_halves(k, positions, mc["rot"])
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    pos_k = list(positions)
    if past is not None:
        k, v, pos_k = torch.cat([past[0], k]), torch.cat([past[1], v]), list(past[2]) + pos_k
    size = int(mc["mask"]["size"]) if mc.get("mask") else 0
    o = sink_attention(q, k, v, chunk_mask(list(positions), pos_k, size), float(mc["scale"]), W[p + "mix.sink"])
    return o.reshape(T, H * dv) @ W[p + "mix.o"].to(F64).T, (k, v, pos_k)


# ---- gated delta rule -------------------------------------------------------------------------------------------------------------------

def short_conv(x, w, before):
    """x [T, C], w [C, taps] (last tap on the current token), before [taps - 1, C] = the inputs of the tokens before -> (y [T, C], the
    last taps - 1 inputs)"""
    x, w = x.to(F64), w.to(F64)
    taps = w.shape[1]
    full = torch.cat([before.to(F64), x])
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + full[j:j + x.shape[0]] * w[:, j]
    return y, full[full.shape[0] - (taps - 1):]


def delta_decay(a_log, dt_bias, a):
    """a [T, H] (the projection) -> g [T, H] in (0, 1)"""
    return torch.exp(-torch.exp(a_log.to(F64)) * softplus(a.to(F64) + dt_bias.to(F64)))


def delta_scan(q, k, v, beta, g, S):
    """q, k [T, H, d] (one per value head), v [T, H, dv], beta, g [T, H], S [H, d, dv] -> (o [T, H, dv], S after the last token)"""
    S = S.to(F64).clone()
    out = []
    for t in range(q.shape[0]):
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def delta_mixer(h, W, p, mc, eps, past=None):
    """past = (conv inputs of q, k, v, S) -> (output [T, width], the same after these tokens)"""
    h = h.to(F64)
    T = h.shape[0]
    H, G, d, dv, taps = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"], mc["conv"]
    if past is None:
        past = (torch.zeros(taps - 1, G * d, dtype=F64), torch.zeros(taps - 1, G * d, dtype=F64), torch.zeros(taps - 1, H * dv, dtype=F64),
                torch.zeros(H, d, dv, dtype=F64))
    conv, tails = {}, []
    for name, before in zip("qkv", past[:3]):
        y, tail = short_conv(h @ W[p + "mix." + name].to(F64).T, W[p + f"mix.{name}.conv"], before)
        conv[name] = silu(y)
        tails.append(tail)
    q = unit_l2(conv["q"].reshape(T, G, d)) * d ** -0.5
    k = unit_l2(conv["k"].reshape(T, G, d))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = sigmoid(h @ W[p + "mix.b"].to(F64).T)
    g = delta_decay(W[p + "mix.A_log"], W[p + "mix.dt_bias"], h @ W[p + "mix.a"].to(F64).T)
    o, S = delta_scan(q, k, conv["v"].reshape(T, H, dv), beta, g, past[3])
    o = unit_rms(o, eps) * W[p + "mix.norm"].to(F64) * silu(h @ W[p + "mix.g"].to(F64).T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ W[p + "mix.o"].to(F64).T, (*tails, S)


# ---- the model -------------------------------------------------------------------------------------------------------------------------

def feed_forward(h, W, p):
    return gelu_exact(h.to(F64) @ W[p + "mlp.up"].to(F64).T) @ W[p + "mlp.down"].to(F64).T


def run_order(cfg):
    """the layer index of every layer run"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


class Model:
    """One sequence: feed() portions of tokens in order. runs_out [layer runs, T, W] is the sum of the streams after every layer run."""

    def __init__(self, cfg, weights):
        self.cfg, self.w = cfg, weights
        self.order = run_order(cfg)
        self.past = [None] * len(self.order)
        self.length = 0

    def feed(self, tokens):
        cfg, W = self.cfg, self.w
        eps = float(cfg["norm"]["eps"])
        pos = list(range(self.length, self.length + len(tokens)))
        x = W["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)]
        X = x[None].repeat(cfg["streams"], 1, 1)
        runs_out = []
        for r, i in enumerate(self.order):
            L, p = cfg["layers"][i], f"l{i}."
            h = layer_norm(streams_read(X, W[p + "hc1.in"]), W[p + "norm1"], eps)
            if L["type"] == "attention":
                y, self.past[r] = attention_mixer(h, W, p, L["mixer"], eps, pos, self.past[r])
            else:
                y, self.past[r] = delta_mixer(h, W, p, L["mixer"], eps, self.past[r])
            X = streams_write(X, y, W[p + "hc1.mix"], W[p + "hc1.out"])
            if L.get("mlp"):
                h = layer_norm(streams_read(X, W[p + "hc2.in"]), W[p + "norm2"], eps)
                X = streams_write(X, feed_forward(h, W, p), W[p + "hc2.mix"], W[p + "hc2.out"])
            runs_out.append(X.sum(dim=0))
        self.length += len(tokens)
        self.runs_out = torch.stack(runs_out)
        return layer_norm(X.sum(dim=0), W["final.norm"], eps) @ W["embed"].to(F64).T


def forward(cfg, weights, tokens):
    """logits [T, vocab] and the streams' sum after every layer run [runs, T, W]"""
    m = Model(cfg, weights)
    logits = m.feed(tokens)
    return logits, m.runs_out


# ---- configurations and random weights of the tests -------------------------------------------------------------------------------------

def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def delta_layer(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": dense(ff)}


def attention_layer(heads, kv_heads, dim, size, ff=None, rot_dims=None, base=1000.0, factor=2.0, scale=None):
    rot_dims = dim if rot_dims is None else rot_dims
    return {"type": "attention", "mlp": dense(ff), "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": size} if size else None,
        "rot": {"base": base, "dims": rot_dims, "scaling": {"factor": factor}}, "scale": dim ** -0.5 if scale is None else scale}}


def make_config(width, vocab, layers, streams=2, loop=None, eps=1e-5):
    cfg = {"architecture": "Relidra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def random_weights(cfg, seed):
    """bf16 tensors of a configuration; decays spread from quick to slow, step sizes and sinks of either sign"""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]

    def rnd(*shape, mean=0.0, spread=1.0):
        return (mean + spread * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    def mat(o, i, gain=1.0):
        return rnd(o, i, spread=gain / math.sqrt(i))

    w = {"embed": rnd(V, W), "final.norm": rnd(W, mean=1.0, spread=0.2)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for q in (1, 2) if L.get("mlp") else (1,):
            w[p + f"norm{q}"] = rnd(W, mean=1.0, spread=0.2)
            w[p + f"hc{q}.in"] = rnd(S, mean=1.0 / S, spread=0.3)
            w[p + f"hc{q}.out"] = rnd(S, mean=0.7, spread=0.3)
            w[p + f"hc{q}.mix"] = (torch.eye(S) * 0.8 + 0.2 * torch.randn(S, S, generator=g)).to(torch.bfloat16)
        if L["type"] == "attention":
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            w[p + "mix.q"], w[p + "mix.q.b"] = mat(H * d, W, 1.5), rnd(H * d, spread=0.5)
            w[p + "mix.k"], w[p + "mix.k.b"] = mat(G * d, W, 1.5), rnd(G * d, spread=0.5)
            w[p + "mix.sink"], w[p + "mix.o"] = rnd(H, mean=0.5), mat(W, H * d)
        else:
            H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for name, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
                w[p + "mix." + name] = mat(c, W, 1.5)
                w[p + f"mix.{name}.conv"] = rnd(c, taps, spread=taps ** -0.5)
            w[p + "mix.g"], w[p + "mix.o"] = mat(H * dv, W, 1.5), mat(W, H * dv)
            w[p + "mix.a"], w[p + "mix.b"] = mat(H, W, 1.5), mat(H, W, 2.0)
            w[p + "mix.A_log"], w[p + "mix.dt_bias"] = rnd(H, mean=-1.0, spread=1.0), rnd(H, mean=-1.0, spread=1.0)
            w[p + "mix.norm"] = rnd(dv, mean=1.0, spread=0.2)
        if L.get("mlp"):
            f = L["mlp"]["ff"]
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(f, W, 1.5), mat(W, f)
    return w
