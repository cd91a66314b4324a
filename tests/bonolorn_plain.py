"""Plain float64 restatement of the Bonolorn design, one function per mechanism, for the tests. It shares no code with the engine.

A model is (cfg, weights): cfg is the config.json tree, weights maps tensor names to torch tensors. x [T, W] is the residual stream of T
tokens of one sequence; no sublayer's input is normed, every sublayer's output is.

  embedding:   x_p = E[token] + pos(p),  pos(p)[2i] = sin(p 10000^(-2i/W)), pos(p)[2i+1] = cos(the same)
  layer:       x <- x + m LN1(mixer(x));  x <- x + m LN2(ff(x));   LN(y) = (y - mean) / sqrt(var + eps) * w
  mixer:       left_scale * attention(x) + right_scale * memory(x)
  attention:   q, k per head unit RMS times a shared weight row; s_ij = scale q_i.k_j - 2^(-8(h+1)/H) (i - j) for 0 <= i - j < size;
               softmax; head h's sum times sigmoid(Wg x)_h; Wo
  memory:      q, k, v = silu(W x); S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; Wo (rms(o over all heads) w * sigmoid(Wg x))
  dense ff:    Wd (gelu_tanh(Wg x) * (Wu x))
  expert:      g = min(Wg x, limit), u = clamp(Wu x, +-limit);  Wd (g sigmoid(1.702 g) (u + 1))
  router:      s = sigmoid(Wr x), choice c = s + correction; a group scores the sum of its two best c; the best `keep` groups stay; of their
               experts the `top` best c; weights s / (sum of the chosen s + 1e-20) * scale; plus one expert that every token uses
  readout:     E . LN(x)
"""
import math

import torch

F64 = torch.float64


def position_vectors(positions, width):
    p = torch.as_tensor(positions, dtype=F64)
    out = torch.zeros(len(positions), width, dtype=F64)
    for c in range(width):
        ang = p * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(ang) if c % 2 == 0 else torch.cos(ang)
    return out


def layer_norm(x, w, eps):
    x = x.to(F64)
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w.to(F64)


def unit_rms(x, eps):
    x = x.to(F64)
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def biased_window_attention(q, k, v, pos_q, pos_k, scale, size):
    """q [Tq, H, d], k [Tk, G, d], v [Tk, G, dv] -> [Tq, H, dv]; size 0: no window"""
    H, G = q.shape[1], k.shape[1]
    dist = torch.as_tensor(pos_q, dtype=F64)[:, None] - torch.as_tensor(pos_k, dtype=F64)[None, :]
    seen = (dist >= 0) & ((dist < size) if size else True)
    out = torch.zeros(q.shape[0], H, v.shape[-1], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h].to(F64) @ k[:, g].to(F64).T) * scale - slope(h, H) * dist
        out[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ v[:, g].to(F64)
    return out


def attention_rows(x, W, p, mc, eps):
    """What the attention keeps per token: normed keys, and values."""
    T = x.shape[0]
    k = unit_rms((x @ W[p + "k"].to(F64).T).reshape(T, mc["kv_heads"], mc["dim"]), eps) * W[p + "k.norm"].to(F64)
    v = (x @ W[p + "v"].to(F64).T).reshape(T, mc["kv_heads"], mc["vdim"])
    return k, v


def attention_mixer(x, W, p, mc, eps, positions, k, v):
    """k, v: rows of positions 0 .. last of the sequence"""
    T = x.shape[0]
    q = unit_rms((x @ W[p + "q"].to(F64).T).reshape(T, mc["heads"], mc["dim"]), eps) * W[p + "q.norm"].to(F64)
    size = mc["mask"]["size"] if mc.get("mask") else 0
    o = biased_window_attention(q, k, v, positions, list(range(k.shape[0])), mc["scale"], size)
    o = o * torch.sigmoid(x @ W[p + "g"].to(F64).T)[:, :, None]
    return o.reshape(T, -1) @ W[p + "o"].to(F64).T


def memory_scan(q, k, v, decay, state):
    """q, k [T, H, d], v [T, H, dv], decay [H], state [H, d, dv] -> (o [T, H, dv], last state)"""
    S = state.to(F64).clone()
    d = torch.as_tensor(decay, dtype=F64)[:, None, None]
    out = torch.zeros(v.shape, dtype=F64)
    for t in range(q.shape[0]):
        S = d * S + k[t].to(F64)[:, :, None] * v[t].to(F64)[:, None, :]
        out[t] = (S * q[t].to(F64)[:, :, None]).sum(dim=1)
    return out, S


def memory_mixer(x, W, p, mc, eps, state):
    T, H = x.shape[0], mc["heads"]
    q, k, v = (silu(x @ W[p + n].to(F64).T).reshape(T, H, -1) for n in "qkv")
    o, last = memory_scan(q, k, v, mc["decay"], state)
    y = unit_rms(o.reshape(T, -1), eps) * W[p + "norm"].to(F64) * torch.sigmoid(x @ W[p + "g"].to(F64).T)
    return y @ W[p + "o"].to(F64).T, last


def dense_ff(x, W, p):
    return (gelu_tanh(x @ W[p + "gate"].to(F64).T) * (x @ W[p + "up"].to(F64).T)) @ W[p + "down"].to(F64).T


def clamped_expert(x, W, p, limit):
    g = torch.clamp(x @ W[p + "gate"].to(F64).T, max=limit)
    u = torch.clamp(x @ W[p + "up"].to(F64).T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].to(F64).T


def choose_experts(z, correction, ro):
    """router logits of one token -> [(expert, weight)], best choice score first"""
    s = [1.0 / (1.0 + math.exp(-float(a))) for a in z]
    c = [a + float(b) for a, b in zip(s, correction)]
    n = len(s)
    allowed = set(range(n))
    if ro.get("groups"):
        count, keep = ro["groups"]["count"], ro["groups"]["keep"]
        size = n // count
        score = [sum(sorted(c[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(count)]
        best = sorted(range(count), key=lambda g: (-score[g], g))[:keep]
        allowed = {e for g in best for e in range(g * size, (g + 1) * size)}
    chosen = sorted(allowed, key=lambda e: (-c[e], e))[:ro["top"]]
    total = sum(s[e] for e in chosen) + 1e-20
    return [(e, s[e] / total * ro["scale"]) for e in chosen]


def moe_ff(x, W, p, ml):
    z = x @ W[p + "router"].to(F64).T
    out = torch.zeros(x.shape[0], W[p + "e0.down"].shape[0], dtype=F64)
    for t in range(x.shape[0]):
        for e, w in choose_experts(z[t], W[p + "correction"], ml["router"]):
            out[t] += w * clamped_expert(x[t:t + 1], W, "%se%d." % (p, e), ml["expert"]["limit"])[0]
    if ml.get("shared"):
        out = out + clamped_expert(x, W, p + "shared.", ml["shared"]["limit"])
    return out


class Model:
    """One sequence: feed() takes its next tokens and returns their logits."""

    def __init__(self, cfg, W):
        self.cfg, self.W, self.pos = cfg, W, 0
        self.layers = []
        for lc in cfg["layers"]:
            A, R = lc["mixer"]["left"], lc["mixer"]["right"]
            self.layers.append({"k": torch.zeros(0, A["kv_heads"], A["dim"], dtype=F64), "v": torch.zeros(0, A["kv_heads"], A["vdim"], dtype=F64),
                                "s": torch.zeros(R["heads"], R["dim"], R["vdim"], dtype=F64)})
        self.runs = []

    def feed(self, tokens):
        cfg, W, eps, m = self.cfg, self.W, self.cfg["norm"]["eps"], self.cfg["residual_mult"]
        positions = list(range(self.pos, self.pos + len(tokens)))
        x = W["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.int64)] + position_vectors(positions, cfg["width"])
        self.runs = []
        for i, lc in enumerate(cfg["layers"]):
            p, st, mc = "l%d." % i, self.layers[i], lc["mixer"]
            k, v = attention_rows(x, W, p + "mix.left.", mc["left"], eps)
            st["k"], st["v"] = torch.cat([st["k"], k]), torch.cat([st["v"], v])
            left = attention_mixer(x, W, p + "mix.left.", mc["left"], eps, positions, st["k"], st["v"])
            right, st["s"] = memory_mixer(x, W, p + "mix.right.", mc["right"], eps, st["s"])
            x = x + m * layer_norm(mc["left_scale"] * left + mc["right_scale"] * right, W[p + "norm1"], eps)
            ml = lc.get("mlp")
            if ml:
                y = dense_ff(x, W, p + "mlp.") if ml["kind"] == "dense" else moe_ff(x, W, p + "mlp.", ml)
                x = x + m * layer_norm(y, W[p + "norm2"], eps)
            self.runs.append(x)
        self.pos += len(tokens)
        return layer_norm(x, W["final.norm"], eps) @ W["embed"].to(F64).T


def forward(cfg, W, tokens):
    """-> (logits [T, vocab], residual stream after every layer [layers, T, width]), float64"""
    m = Model(cfg, W)
    logits = m.feed(list(tokens))
    return logits, torch.stack(m.runs) if m.runs else torch.zeros(0)


# ---- small configurations and random weights for the tests ----------------------------------------------------------------------------
def dense_mlp(ff):
    return {"kind": "dense", "ff": ff}


def moe_mlp(ff, experts, top, groups=(1, 1), scale=1.0, limit=2.0, shared=None, shared_limit=None):
    ml = {"kind": "moe", "expert": {"ff": ff, "limit": float(limit)},
          "router": {"experts": experts, "top": top, "scale": float(scale), "groups": {"count": groups[0], "keep": groups[1]}}}
    if shared:
        ml["shared"] = {"ff": shared, "limit": float(limit if shared_limit is None else shared_limit)}
    return ml


def layer(heads, kv_heads, dim, vdim, size, r_heads, r_dim, r_vdim, decay, mlp=None, scale=None, left_scale=1.0, right_scale=1.0):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(dim ** -0.5 if scale is None else scale), "mask": {"size": size}}
    right = {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": [float(d) for d in decay]}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": float(left_scale), "right": right, "right_scale": float(right_scale)}, "mlp": mlp}


def make_config(width, vocab, layers, eps=1e-5, residual_mult=0.6):
    return {"architecture": "Bonolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": residual_mult, "layers": layers}


def random_weights(cfg, seed=0):
    """bf16 tensors (what a checkpoint holds), as a dict of torch tensors"""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(rows, cols, gain=1.0):
        return (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(torch.bfloat16)

    def vec(n, mean=0.0, spread=0.1):
        return (mean + spread * torch.randn(n, generator=g)).to(torch.bfloat16)

    def expert(p, f):
        t[p + "gate"], t[p + "up"], t[p + "down"] = mat(f, W, 1.3), mat(f, W, 1.3), mat(W, f)

    t = {"embed": mat(V, W, math.sqrt(W)), "final.norm": vec(W, 1.0, 0.2)}
    for i, lc in enumerate(cfg["layers"]):
        p, A, R = "l%d." % i, lc["mixer"]["left"], lc["mixer"]["right"]
        H, G, D, Dv = A["heads"], A["kv_heads"], A["dim"], A["vdim"]
        l, r = p + "mix.left.", p + "mix.right."
        t[p + "norm1"] = vec(W, 1.0, 0.2)
        t[l + "q"], t[l + "k"], t[l + "v"] = mat(H * D, W), mat(G * D, W), mat(G * Dv, W)
        t[l + "q.norm"], t[l + "k.norm"] = vec(D, 1.3, 0.3), vec(D, 1.3, 0.3)
        t[l + "g"], t[l + "o"] = mat(H, W, 1.5), mat(W, H * Dv, 1.5)
        Hr, Dr, Dvr = R["heads"], R["dim"], R["vdim"]
        t[r + "q"], t[r + "k"], t[r + "v"] = mat(Hr * Dr, W), mat(Hr * Dr, W), mat(Hr * Dvr, W)
        t[r + "g"], t[r + "o"], t[r + "norm"] = mat(Hr * Dvr, W, 1.5), mat(W, Hr * Dvr, 1.5), vec(Hr * Dvr, 1.0, 0.3)
        ml = lc.get("mlp")
        if not ml:
            continue
        t[p + "norm2"] = vec(W, 1.0, 0.2)
        if ml["kind"] == "dense":
            expert(p + "mlp.", ml["ff"])
        else:
            E = ml["router"]["experts"]
            t[p + "mlp.router"], t[p + "mlp.correction"] = mat(E, W, 1.5), vec(E, -0.3, 0.3)
            for x in range(E):
                expert("%smlp.e%d." % (p, x), ml["expert"]["ff"])
            if ml.get("shared"):
                expert(p + "mlp.shared.", ml["shared"]["ff"])
    return t
