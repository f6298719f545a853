"""Oracle for the Nosolix design (a layer list of selective scans and of windowed attention beside a state-space dual
recurrence, Dynamic Tanh in the place of norms, sigmoid-routed clamped experts beside a gated shared one): plain, slow
float64 PyTorch, one function per mechanism.

TEST INFRASTRUCTURE.  Nothing here is shared with the product path.  Notation: t / j are positions from 0, W matrices
are [out, in] and act as h @ W.T, n(z, g) = z / sqrt(mean(z^2) + eps) * g, conv is causal per channel.

  embedding    x_t = E[tok_t] * scale
  layer        x <- x + mixer(dyt1(x));  x <- x + ff(dyt2(x)),  dyt(x) = tanh(alpha x) * w + b
  mamba1       [x~ | z] = h Win;  u = silu(conv(x~) + bc);  [r | B | C] = u Wx;  D_t = softplus(r Wdt + bdt) per channel;
               S[c, n] <- exp(-D_t[c] exp(A_log[c, n])) S[c, n] + D_t[c] u[c] B[n];  y[c] = sum_n S[c, n] C[n] + D[c] u[c];
               (y * silu(z)) Wo
  parallel     left: heads on fewer key / value heads, the first `dims` numbers of q and k turn in pairs (i, i + dims / 2) by
               t f_i;  softmax over j with 0 <= t - j < size of scale q.k;  (heads side by side * sigmoid(h Wg)) Wo
               right: [z | x~ | B~ | C~ | r] = h Win;  [x | B | C] = silu(conv(.) + bc);  D_t = softplus(r + dt_bias) per head;
               S <- exp(-D_t exp(A_log)) S + D_t B x^T;  y = S^T C + D x (B, C shared by the heads of a group);
               (n(y * silu(z)) in equal parts * g) Wo
               result: (n(left, g_left) + n(right, g_right)) / 2
  frequencies  f_i = base^(-2i/dims); with wavelength l = 2 pi / f: l < original / high - f;  l > original / low - f / factor;
               between - (1 - s) f / factor + s f with s = (original / l - low) / (high - low)
  dense        relu(h Wu)^2 Wd
  moe          s = sigmoid(h Wr), c = s + correction; neighbours form equal groups, the `keep` with the largest sum of their
               two best c stay, the `top` largest c among them are chosen; weights s / (sum s + 1e-20) * scale;
               expert(h): g = min(h Wg, limit), u = clamp(h Wu, +-limit), (g sigmoid(1.702 g) (u + 1)) Wd;
               + sigmoid(h . sg) * shared(h)
  logits       dyt_final(x) head^T
"""
from __future__ import annotations

import math

import torch

from .hybrid import DT, save_model_dir  # noqa: F401  (file writer only: config.json + safetensors by hand)


def moe_mlp(ff=12, limit=1.5, experts=6, top=3, groups=2, keep=1, scale=1.75, shared_ff=10, shared_limit=0.75):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "groups": {"count": groups, "keep": keep}, "scale": scale, "top": top}}
    if shared_ff:
        f["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return f


def dense_mlp(ff=20):
    return {"kind": "dense", "ff": ff}


def mamba_layer(inner=20, state=6, dt_rank=3, conv=4, mlp="default"):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}, "mlp": moe_mlp() if mlp == "default" else mlp}


def parallel_layer(heads=4, kv_heads=2, dim=8, vdim=6, size=7, scale=0.3, base=400.0, dims=None, factor=4.0, low=1.0, high=4.0, original=40,
                   r_heads=4, r_vdim=5, state=6, groups=2, norm_groups=2, conv=3, mlp="default"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale,
            "rot": {"base": base, "dims": dim if dims is None else dims, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}}
    right = {"heads": r_heads, "vdim": r_vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": moe_mlp() if mlp == "default" else mlp}


def make_config(layers, vocab=97, width=24, eps=1e-5, scale=3.0):
    return {"architecture": "Nosolix", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def tensor_shapes(cfg):
    D, V = cfg["width"], cfg["vocab"]
    sh = {"embed": (V, D), "head": (V, D)}

    def norm(name):
        sh.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})

    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for z in ("norm1",) + (("norm2",) if L["mlp"] else ()):
            norm(p + z)
        x = p + "mix."
        if L["type"] == "mamba1":
            I, N, R = m["inner"], m["state"], m["dt_rank"]
            sh.update({x + "in": (2 * I, D), x + "conv": (I, m["conv"]), x + "conv.b": (I,), x + "x": (R + 2 * N, I), x + "dt": (I, R), x + "dt.b": (I,),
                       x + "A_log": (I, N), x + "D": (I,), x + "o": (D, I)})
        else:
            a, r = m["left"], m["right"]
            nv, I, C = a["heads"] * a["vdim"], r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
            y, z = x + "left.", x + "right."
            sh.update({y + "q": (a["heads"] * a["dim"], D), y + "k": (a["kv_heads"] * a["dim"], D), y + "v": (a["kv_heads"] * a["vdim"], D), y + "g": (nv, D), y + "o": (D, nv),
                       y + "out": (D,), z + "in": (I + C + r["heads"], D), z + "conv": (C, r["conv"]), z + "conv.b": (C,), z + "dt_bias": (r["heads"],),
                       z + "A_log": (r["heads"],), z + "D": (r["heads"],), z + "norm": (I,), z + "o": (D, I), z + "out": (D,)})
        f = L["mlp"]
        q = p + "mlp."
        if f and f["kind"] == "dense":
            sh.update({q + "up": (f["ff"], D), q + "down": (D, f["ff"])})
        elif f:
            E = f["router"]["experts"]
            sh.update({q + "router": (E, D), q + "correction": (E,)})
            for e in range(E):
                sh.update({f"{q}e{e}.gate": (f["expert"]["ff"], D), f"{q}e{e}.up": (f["expert"]["ff"], D), f"{q}e{e}.down": (D, f["expert"]["ff"])})
            if f.get("shared"):
                n = f["shared"]["ff"]
                sh.update({q + "shared.gate": (n, D), q + "shared.up": (n, D), q + "shared.down": (D, n), q + "shared.sg": (1, D)})
    return sh


def make_weights(cfg, seed=0):
    """Random bfloat16-representable weights (returned as float64) sized so that activations stay O(1), step sizes and decays
    spread widely, Dynamic Tanh bends and shifts its input, and corrections (of both signs) change choices."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        parts = name.split(".")
        last, owner = parts[-1], parts[-2] if len(parts) > 1 else ""
        r = lambda s=1.0: s * torch.randn(shape, generator=g)
        if last in ("norm", "norm1", "norm2", "out"):
            t = 1.0 + 0.3 * r()
        elif last == "alpha":
            t = 0.5 + 0.3 * torch.rand(shape, generator=g)
        elif last == "b" and owner in ("norm", "norm1", "norm2"):
            t = r(0.2)
        elif last == "b" and owner == "conv":
            t = r(0.3)
        elif last == "b" or last == "dt_bias":
            t = r(1.0) - 1.0
        elif last == "conv":
            t = 0.5 * r() + (torch.arange(shape[1]) == shape[1] - 1).to(torch.float32)
        elif last == "embed":
            t = r(0.4)
        elif last == "A_log":
            t = r(0.8) - 0.5
        elif last == "D":
            t = 1.0 + r(0.5)
        elif last == "correction":
            t = r(0.3) - 0.4
        elif last == "dt":
            t = r(1.0 / math.sqrt(shape[-1]))
        elif last in ("o", "down") and len(parts) > 2 and "left" not in parts and "right" not in parts:
            t = r(0.4 / math.sqrt(shape[-1]))      # results that are not normed before they join the stream
        else:
            t = r(1.5 / math.sqrt(shape[-1]))
        W[name] = t.to(torch.bfloat16).to(DT)
    return W


# ------------------------------------------------------------------------------------------ mechanisms

ROUND = None      # a function applied to every stored activation: None for the exact oracle; see bfloat16_noise()


def _r(t):
    return t if ROUND is None else ROUND(t)


def bfloat16_noise(cfg, W, tokens):
    """Per position, the size (root mean square over the vocabulary, relative to the logits' size) of what rounding alone
    does: the distance between the oracle and the oracle with every stored activation - sublayer inputs, projection and
    convolution outputs, cached keys and values, gated products, sublayer results - rounded to bfloat16 once."""
    global ROUND
    exact = forward(cfg, W, tokens)
    ROUND = lambda t: t.to(torch.bfloat16).to(DT)
    try:
        noisy = forward(cfg, W, tokens)
    finally:
        ROUND = None
    return ((noisy - exact).pow(2).mean(-1).sqrt() / exact.pow(2).mean().sqrt()).numpy()


def float32_noise(cfg, W, tokens):
    """The same for 32-bit arithmetic: the distance between the oracle and its equations evaluated in float32."""
    exact, single = forward(cfg, W, tokens), forward(cfg, {k: v.to(torch.float32) for k, v in W.items()}, tokens)
    return ((single - exact).pow(2).mean(-1).sqrt() / exact.pow(2).mean().sqrt()).numpy()


silu = torch.nn.functional.silu
softplus = lambda z: torch.logaddexp(z, torch.zeros_like(z))


def rms(z, eps, g=None):
    y = z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps)
    return y if g is None else y * g


def dyt(x, W, name):
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def short_conv(u, w, b):
    """u [T, C]; w [C, taps]: y_t = b + sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = b.expand_as(u).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def selective_scan(u, D, A, B, C):
    """u, D [T, I]; A [I, N]; B, C [T, N] -> (y [T, I] without the direct term, final state [I, N])"""
    S = torch.zeros_like(A)
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = torch.exp(D[t][:, None] * A) * S + (D[t] * u[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t]
    return y, S


def mamba1(h, P, m):
    I, N, R = m["inner"], m["state"], m["dt_rank"]
    xz = _r(h @ P["in"].T)
    u = _r(silu(short_conv(xz[:, :I], P["conv"], P["conv.b"])))
    rbc = _r(u @ P["x"].T)
    D = softplus(rbc[:, :R] @ P["dt"].T + P["dt.b"])
    y, _ = selective_scan(u, D, -torch.exp(P["A_log"]), rbc[:, R:R + N], rbc[:, R + N:])
    return _r(_r((y + P["D"] * u) * silu(xz[:, I:])) @ P["o"].T)


def frequencies(rot):
    n, s = rot["dims"], rot.get("scaling")
    out = []
    for i in range(n // 2):
        f = rot["base"] ** (-2.0 * i / n)
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                k = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - k) * f / s["factor"] + k * f
        out.append(f)
    return out


def turn(x, rot):
    """x [T, heads, dim] at positions 0 .. T - 1: the first `dims` numbers in pairs (i, i + dims / 2)."""
    n = rot["dims"] // 2
    if n == 0:
        return x
    a = torch.arange(x.shape[0], dtype=DT)[:, None, None] * torch.tensor(frequencies(rot), dtype=DT)
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[:, :, :n], x[:, :, n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[:, :, 2 * n:]], dim=-1)


def attention_weights(h, P, m):
    """softmax weights [heads, T, T]"""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = _r(turn(_r(h @ P["q"].T).reshape(T, H, m["dim"]), m["rot"]))
    k = _r(turn(_r(h @ P["k"].T).reshape(T, G, m["dim"]), m["rot"]))
    t, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    s = torch.einsum("thd,jhd->htj", q, k[:, torch.arange(H) // (H // G)]) * m["scale"]
    return torch.softmax(s.masked_fill(~((t - j >= 0) & (t - j < m["mask"]["size"])), -math.inf), dim=-1)


def attention(h, P, m):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    v = _r(h @ P["v"].T).reshape(T, G, m["vdim"])
    o = _r(torch.einsum("htj,jhv->thv", attention_weights(h, P, m), v[:, torch.arange(H) // (H // G)]).reshape(T, -1))
    return _r(_r(o * torch.sigmoid(_r(h @ P["g"].T))) @ P["o"].T)


def dual_scan(x, B, C, a, D):
    """x [T, H, P]; B, C [T, G, N]; a (decay), D (step) [T, H] -> (y [T, H, P] without the direct term, final state [H, N, P])"""
    T, H, G = x.shape[0], x.shape[1], B.shape[1]
    g = torch.arange(H) // (H // G)
    S = torch.zeros(H, B.shape[2], x.shape[2], dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        S = a[t][:, None, None] * S + D[t][:, None, None] * B[t, g][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, C[t, g])
    return y, S


def mamba2(h, P, m, eps):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    I, GN = H * V, G * N
    p = _r(h @ P["in"].T)
    z, r = p[:, :I], p[:, 2 * I + 2 * GN:]
    xbc = _r(silu(short_conv(p[:, I:2 * I + 2 * GN], P["conv"], P["conv.b"])))
    x, B, C = xbc[:, :I].reshape(T, H, V), xbc[:, I:I + GN].reshape(T, G, N), xbc[:, I + GN:].reshape(T, G, N)
    D = softplus(r + P["dt_bias"])
    y, _ = dual_scan(x, B, C, torch.exp(-torch.exp(P["A_log"]) * D), D)
    y = (y + P["D"][:, None] * x).reshape(T, I) * silu(z)
    y = rms(y.reshape(T, m["norm_groups"], -1), eps).reshape(T, I) * P["norm"]
    return _r(_r(y) @ P["o"].T)


def parallel(h, P, m, eps):
    a, b = sub(P, "left."), sub(P, "right.")
    return 0.5 * (rms(attention(h, a, m["left"]), eps, a["out"]) + rms(mamba2(h, b, m["right"], eps), eps, b["out"]))


def group_scores(c, G):
    """sum of the two largest choice scores of every group, [T, G]"""
    return torch.sort(c.reshape(c.shape[0], G, -1), dim=-1, descending=True).values[:, :, :2].sum(-1)


def route(h, P, r):
    """(chosen [T, top] in falling order of the choice score, their weights [T, top])"""
    s = torch.sigmoid(h @ P["router"].T)
    c = s + P["correction"]
    n, G = s.shape[1], r["groups"]["count"]
    best = group_scores(c, G)
    kept = torch.zeros(h.shape[0], G, dtype=torch.bool)
    for _ in range(r["groups"]["keep"]):
        i = torch.argmax(best.masked_fill(kept, -math.inf), dim=1)
        kept[torch.arange(h.shape[0]), i] = True
    c = c.masked_fill(~kept.repeat_interleave(n // G, dim=1), -math.inf)
    chosen = torch.sort(c, dim=1, descending=True, stable=True).indices[:, :r["top"]]
    w = torch.gather(s, 1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def route_margin(h, P, r):
    """How close a token's choice is: the smallest gap between the choice scores of the last chosen and the first left out
    expert, or between the scores of the last kept and the first dropped group."""
    c = torch.sigmoid(h @ P["router"].T) + P["correction"]
    T, n, G, K = h.shape[0], c.shape[1], r["groups"]["count"], r["groups"]["keep"]
    best = group_scores(c, G)
    order = torch.sort(best, dim=1, descending=True).values
    gap = order[:, K - 1] - order[:, K] if K < G else torch.full((T,), math.inf, dtype=DT)
    kept = best >= order[:, K - 1:K]
    cs = torch.sort(c.masked_fill(~kept.repeat_interleave(n // G, dim=1), -math.inf), dim=1, descending=True).values
    if r["top"] < n // G * K:
        gap = torch.minimum(gap, cs[:, r["top"] - 1] - cs[:, r["top"]])
    return gap


def clamped_unit(h, P, e, limit):
    g = torch.clamp(h @ P[e + ".gate"].T, max=limit)
    u = torch.clamp(h @ P[e + ".up"].T, -limit, limit)
    return _r(_r(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ P[e + ".down"].T)


def moe(h, P, f):
    chosen, w = route(h, P, f["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), w[t]):
            out[t] += s * clamped_unit(h[t], P, f"e{e}", f["expert"]["limit"])
    if f.get("shared"):
        out = out + torch.sigmoid(h @ P["shared.sg"].T) * clamped_unit(h, P, "shared", f["shared"]["limit"])
    return out


def dense(h, P):
    return _r(_r(torch.relu(h @ P["up"].T).pow(2)) @ P["down"].T)


def sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(cfg, W, tokens, return_layers=False, margins=None):
    """Logits [T, vocab] of one sequence (float64); optionally the residual stream after every layer.  margins (a list)
    receives every layer's route_margin."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    layers = []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        P = sub(W, p + "mix.")
        h = _r(dyt(x, W, p + "norm1"))
        x = x + (mamba1(h, P, m) if L["type"] == "mamba1" else parallel(h, P, m, eps))
        f = L["mlp"]
        if f:
            h = _r(dyt(x, W, p + "norm2"))
            M = sub(W, p + "mlp.")
            if f["kind"] == "dense":
                x = x + dense(h, M)
            else:
                if margins is not None:
                    margins.append(route_margin(h, M, f["router"]))
                x = x + moe(h, M, f)
        layers.append(x.clone())
    logits = _r(_r(dyt(x, W, "final.norm")) @ W["head"].T)
    return (logits, layers) if return_layers else logits


def greedy(cfg, W, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]
