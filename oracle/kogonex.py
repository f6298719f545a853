"""Oracle for the Kogonex design (a layer list of latent attention with a window, sinks and shared latents, and of a gated
delta rule with a decay per key channel, norms on the sublayers' outputs only): plain, slow float64 PyTorch, one function
per mechanism.

TEST INFRASTRUCTURE.  Nothing here is shared with the product path.  Notation: t / j are positions from 0, W matrices
are [out, in] and act as h @ W.T, n(z, g) = z / sqrt(mean(z^2) + eps) * g.

  embedding    x_t = E[tok_t] + B[(tok_(t-1) mul_prev + tok_t mul_cur) mod buckets];  t = 0 takes row `buckets` of B
  layer        x <- x + n(mixer(x), g1);  x <- x + n(moe(x), g2)
  latent       [c~ | r~] = h Wdkv;  c = n(c~, g_kv), r = turn(r~);  per head q = [q' | turn(q'')] of h Wq, key [c Wuk | r], value
               c Wuv;  t sees j with 0 <= t - j < size;  weights e^s / (sum e^s + e^sink), s = scale q.k;  then Wo.  A layer with
               kv_from takes c and r of that layer and has no Wdkv.  turn: pairs (2i, 2i + 1) by t f_i, times m, where
               (YaRN) f_i = base^(-2i/n) (ramp_i / factor + 1 - ramp_i), m = 0.1 ln(factor) + 1
  delta        q, k, v = silu(conv(h Wz)) per channel;  q, k <- z / sqrt(sum z^2 + 1e-6) per head, q also / sqrt(dim);
               beta = sigmoid(h Wb) per head;  a = exp(-exp(A_log) softplus(h Wa1 Wa2 + dt)) per head and key channel;
               per head S <- diag(a_t) S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t (S from zero);
               (n(o, g) per head) * sigmoid(h Wg1 Wg2), then Wo.  Several heads may read one q / k head.
  moe          s = softmax(h Wr) over experts and identity experts;  c = s + correction;  neighbours form equal groups, the
               `keep` groups with the largest best c stay;  the `top` largest c among them are chosen;  sum of s_e expert_e(h)
               with expert(h) = (silu(h Wg) * (h Wu)) Wd, and h itself for an identity expert
  logits       n(x, g_final) head^T
"""
from __future__ import annotations

import math

import torch

from .hybrid import DT, save_model_dir  # noqa: F401  (file writer only: config.json + safetensors by hand)


def moe_mlp(ff=12, experts=6, identity=2, top=3, groups=2, keep=1):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "groups": {"count": groups, "keep": keep}, "identity": identity, "top": top}}


def latent_layer(heads=3, dim=8, rot_dim=4, vdim=6, kv_rank=10, size=7, scale=0.15, base=500.0, factor=4.0, original=64, fast=6.0, slow=1.0, kv_from=None,
                 mlp="default"):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": size}, "scale": scale,
         "rot": {"base": base, "dims": rot_dim, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": moe_mlp() if mlp == "default" else mlp}


def delta_layer(heads=4, kv_heads=2, dim=8, vdim=6, conv=3, mlp="default"):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": moe_mlp() if mlp == "default" else mlp}


def make_config(layers, vocab=97, width=24, eps=1e-5, buckets=53, mul_prev=13, mul_cur=29):
    return {"architecture": "Kogonex", "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": layers,
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


def tensor_shapes(cfg, decay_rank=5, gate_rank=7):
    D, V = cfg["width"], cfg["vocab"]
    sh = {"embed": (V, D), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, D), "final.norm": (D,), "head": (V, D)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for z in ("norm1",) + (("norm2",) if L["mlp"] else ()):
            sh[p + z] = (D,)
        x = p + "mix."
        if L["type"] == "latent_attention":
            H = m["heads"]
            sh[x + "q"] = (H * (m["dim"] + m["rot_dim"]), D)
            if m.get("kv_from") is None:
                sh.update({x + "dkv": (m["kv_rank"] + m["rot_dim"], D), x + "dkv.norm": (m["kv_rank"],)})
            sh.update({x + "uk": (H * m["dim"], m["kv_rank"]), x + "uv": (H * m["vdim"], m["kv_rank"]), x + "sink": (H,), x + "o": (D, H * m["vdim"])})
        else:
            H, nk, nv = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for z, n in (("q", nk), ("k", nk), ("v", nv)):
                sh.update({x + z: (n, D), x + z + ".conv": (n, m["conv"])})
            sh.update({x + "b": (H, D), x + "A_log": (H,), x + "dt_bias": (H * m["dim"],), x + "a1": (decay_rank, D), x + "a2": (H * m["dim"], decay_rank),
                       x + "g1": (gate_rank, D), x + "g2": (nv, gate_rank), x + "norm": (m["vdim"],), x + "o": (D, nv)})
        f = L["mlp"]
        if f:
            r = f["router"]
            sh[p + "mlp.router"] = (r["experts"] + r["identity"], D)
            sh[p + "mlp.correction"] = (r["experts"] + r["identity"],)
            for e in range(r["experts"]):
                sh.update({f"{p}mlp.e{e}.gate": (f["expert"]["ff"], D), f"{p}mlp.e{e}.up": (f["expert"]["ff"], D), f"{p}mlp.e{e}.down": (D, f["expert"]["ff"])})
    return sh


def make_weights(cfg, seed=0, decay_rank=5, gate_rank=7):
    """Random bfloat16-representable weights (returned as float64) sized so that activations stay O(1), decays spread over
    (0, 1), sinks take a visible share and corrections (of both signs) change choices."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg, decay_rank, gate_rank).items():
        last = name.split(".")[-1]
        r = lambda s=1.0: s * torch.randn(shape, generator=g)
        if last in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.3 * r()
        elif last == "conv":
            t = 0.5 * r() + (torch.arange(shape[1]) == shape[1] - 1).to(torch.float32)
        elif name in ("embed", "bigram"):
            t = r(0.8)
        elif last == "sink":
            t = r(1.0) + 1.0
        elif last == "A_log":
            t = r(0.7) - 1.0
        elif last == "dt_bias":
            t = r(1.5) - 1.0
        elif last == "correction":
            t = r(0.15) - 0.1
        elif last == "router":
            t = r(1.5 / math.sqrt(shape[-1]))
        elif last == "a2":
            t = r(2.0 / math.sqrt(shape[-1]))
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
    convolution outputs, cached latents, gated products, sublayer results - rounded to bfloat16 once."""
    global ROUND
    exact = forward(cfg, W, tokens)
    ROUND = lambda t: t.to(torch.bfloat16).to(DT)
    try:
        noisy = forward(cfg, W, tokens)
    finally:
        ROUND = None
    return ((noisy - exact).pow(2).mean(-1).sqrt() / exact.pow(2).mean().sqrt()).numpy()


def rms(z, eps, g=None):
    y = z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps)
    return y if g is None else y * g


def bigram_rows(tokens, b):
    return [b["buckets"] if t == 0 else (tokens[t - 1] * b["mul_prev"] + tokens[t] * b["mul_cur"]) % b["buckets"] for t in range(len(tokens))]


def embedding(tokens, W, b):
    return W["embed"][torch.tensor(tokens)] + W["bigram"][torch.tensor(bigram_rows(tokens, b))]


def short_conv(u, w):
    """u [T, C]; w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def yarn(rot):
    """(frequencies [dims / 2], multiplier of cos and sin)"""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    at = lambda t: n * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def turn(x, positions, rot):
    """x [T, dims]: interleaved pairs."""
    if rot["dims"] == 0:
        return x
    f, mult = yarn(rot)
    a = torch.as_tensor(positions, dtype=DT)[:, None] * torch.tensor(f, dtype=DT)[None, :]
    c, s = mult * torch.cos(a), mult * torch.sin(a)
    u, v = x[:, 0::2], x[:, 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], dim=-1).reshape(x.shape)


def latents(h, P, m, eps):
    """(normed latent [T, kv_rank], turned shared key part [T, rot_dim]): what a layer caches."""
    z = _r(h @ P["dkv"].T)
    c = _r(rms(z[:, :m["kv_rank"]], eps, P["dkv.norm"]))
    return c, _r(turn(z[:, m["kv_rank"]:], list(range(h.shape[0])), m["rot"]))


def window_visible(t, j, size):
    return 0 <= t - j < size


def sink_softmax(s, vis, sink):
    """softmax weights over the visible scores, with e^sink in the denominator"""
    s = s.masked_fill(~vis, -math.inf)
    mx = torch.maximum(s.max(-1, keepdim=True).values, torch.as_tensor(sink, dtype=DT))
    e = torch.exp(s - mx)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - mx))


def latent_weights(h, P, m, c, r, head):
    """softmax weights [T, T] of one head"""
    T, d, n = h.shape[0], m["dim"], m["rot_dim"]
    q = _r(h @ P["q"].T).reshape(T, m["heads"], d + n)[:, head]
    qr = _r(turn(q[:, d:], list(range(T)), m["rot"]))
    k = _r(c @ P["uk"][head * d:(head + 1) * d].T)
    s = (q[:, :d] @ k.T + qr @ r.T) * m["scale"]
    t, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return sink_softmax(s, (t - j >= 0) & (t - j < m["mask"]["size"]), P["sink"][head])


def latent_attention(h, P, m, c, r):
    out = []
    for i in range(m["heads"]):
        w = latent_weights(h, P, m, c, r, i)
        out.append(w @ _r(c @ P["uv"][i * m["vdim"]:(i + 1) * m["vdim"]].T))
    return _r(_r(torch.cat(out, dim=-1)) @ P["o"].T)


def unit(z):
    return z / torch.sqrt(z.pow(2).sum(-1, keepdim=True) + 1e-6)


def delta_decay(h, P, m):
    z = _r(h @ P["a1"].T) @ P["a2"].T + P["dt_bias"]
    sp = torch.nn.functional.softplus(z).reshape(h.shape[0], m["heads"], m["dim"])
    return torch.exp(-torch.exp(P["A_log"])[None, :, None] * sp)


def delta_inputs(h, P, m):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    act = lambda z: _r(torch.nn.functional.silu(short_conv(_r(h @ P[z].T), P[z + ".conv"])))
    q, k, v = act("q").reshape(T, G, m["dim"]), act("k").reshape(T, G, m["dim"]), act("v").reshape(T, H, m["vdim"])
    return unit(q) / math.sqrt(m["dim"]), unit(k), v, torch.sigmoid(_r(h @ P["b"].T)), delta_decay(h, P, m)


def delta_scan(q, k, v, beta, a):
    """q, k [T, G, dim], v [T, H, vdim], beta [T, H], a [T, H, dim] -> (o [T, H, vdim], final state [H, dim, vdim])"""
    T, H, G = v.shape[0], v.shape[1], q.shape[1]
    hk = torch.arange(H) // (H // G)
    S = torch.zeros(H, q.shape[2], v.shape[2], dtype=DT)
    o = torch.zeros_like(v)
    for t in range(T):
        S = a[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t, hk]))
        S = S + k[t, hk][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t, hk])
    return o, S


def channel_delta(h, P, m, eps, return_state=False):
    T = h.shape[0]
    o, S = delta_scan(*delta_inputs(h, P, m))
    gate = torch.sigmoid(_r(_r(h @ P["g1"].T) @ P["g2"].T))
    y = _r(rms(o, eps, P["norm"]).reshape(T, -1) * gate)
    out = _r(y @ P["o"].T)
    return (out, S) if return_state else out


def route(h, P, r):
    """(chosen [T, top] in falling order of the choice score, their weights [T, top])"""
    s = torch.softmax(h @ P["router"].T, dim=-1)
    c = s + P["correction"]
    n, G = s.shape[1], r["groups"]["count"]
    best = c.reshape(-1, G, n // G).max(-1).values
    kept = torch.zeros(h.shape[0], G, dtype=torch.bool)
    for _ in range(r["groups"]["keep"]):
        i = torch.argmax(best.masked_fill(kept, -math.inf), dim=1)
        kept[torch.arange(h.shape[0]), i] = True
    c = c.masked_fill(~kept.repeat_interleave(n // G, dim=1), -math.inf)
    chosen = torch.sort(c, dim=1, descending=True, stable=True).indices[:, :r["top"]]
    return chosen, torch.gather(s, 1, chosen)


def route_margin(h, P, r):
    """How close a token's choice is: the smallest gap between two choice scores (of the last chosen and the first left out
    expert, or of the best ones of the last kept and the first dropped group), relative to the larger of the two scores."""
    s = torch.softmax(h @ P["router"].T, dim=-1)
    c = s + P["correction"]
    T, n, G, K = h.shape[0], s.shape[1], r["groups"]["count"], r["groups"]["keep"]
    rel = lambda ca, cb, sa, sb: (ca - cb) / torch.maximum(sa, sb)
    best, arg = c.reshape(T, G, n // G).max(-1)
    sbest = torch.gather(s.reshape(T, G, n // G), 2, arg[:, :, None])[:, :, 0]
    order = torch.sort(best, dim=1, descending=True).indices
    at = lambda t, k: torch.gather(t, 1, order[:, k:k + 1])[:, 0]
    gap = rel(at(best, K - 1), at(best, K), at(sbest, K - 1), at(sbest, K)) if K < G else torch.full((T,), math.inf, dtype=DT)
    kept = best >= at(best, K - 1)[:, None]
    order = torch.sort(c.masked_fill(~kept.repeat_interleave(n // G, dim=1), -math.inf), dim=1, descending=True).indices
    if r["top"] < n // G * K:
        k = r["top"]
        gap = torch.minimum(gap, rel(at(c, k - 1), at(c, k), at(s, k - 1), at(s, k)))
    return gap


def expert(h, P, e):
    return _r(_r(torch.nn.functional.silu(h @ P[f"e{e}.gate"].T) * (h @ P[f"e{e}.up"].T)) @ P[f"e{e}.down"].T)


def moe(h, P, f):
    r = f["router"]
    chosen, w = route(h, P, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), w[t]):
            out[t] += s * (h[t] if e >= r["experts"] else expert(h[t], P, e))
    return out


def sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(cfg, W, tokens, return_layers=False, margins=None):
    """Logits [T, vocab] of one sequence (float64); optionally the residual stream after every layer.  margins (a list)
    receives every layer's route_margin."""
    eps = cfg["norm"]["eps"]
    x = embedding(tokens, W, cfg["embedding"]["bigram"])
    layers, cached = [], {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        P = sub(W, p + "mix.")
        h = _r(x)
        if L["type"] == "latent_attention":
            if m.get("kv_from") is None:
                cached[i] = latents(h, P, m, eps)
            y = latent_attention(h, P, m, *cached[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            y = channel_delta(h, P, m, eps)
        x = x + rms(y, eps, W[p + "norm1"])
        if L["mlp"]:
            h = _r(x)
            M = sub(W, p + "mlp.")
            if margins is not None:
                margins.append(route_margin(h, M, L["mlp"]["router"]))
            x = x + rms(moe(h, M, L["mlp"]), eps, W[p + "norm2"])
        layers.append(x.clone())
    logits = _r(_r(rms(x, eps, W["final.norm"])) @ W["head"].T)
    return (logits, layers) if return_layers else logits


def greedy(cfg, W, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]
