"""Host-side pieces of the Nosolix design: the config reader (every size and constant from config.json, refusals) and the
oracle's own mechanisms against closed forms."""
import ctypes as C
import json
import math

import torch

from oracle import nosolix as ok


def spec_of(kge, path):
    L = kge.lib()
    h = L.kge_model_open(str(path).encode())
    assert h, L.kge_last_error()
    buf = C.create_string_buffer(1 << 16)
    assert L.kge_model_spec_json(h, buf, 1 << 16) > 0
    L.kge_model_close(h)
    return json.loads(buf.value)


def test_config_reader_takes_every_size_and_constant(kge, tmp_path):
    layers = [ok.mamba_layer(inner=26, state=9, dt_rank=5, conv=3, mlp=ok.dense_mlp(34)),
              ok.parallel_layer(heads=6, kv_heads=3, dim=10, vdim=7, size=19, scale=0.41, base=777.0, dims=6, factor=3.0, low=1.5, high=5.0, original=100,
                                r_heads=8, r_vdim=3, state=11, groups=4, norm_groups=6, conv=5,
                                mlp=ok.moe_mlp(ff=9, limit=1.25, experts=12, top=5, groups=4, keep=2, scale=1.5, shared_ff=14, shared_limit=0.5)),
              ok.mamba_layer(mlp=None)]
    cfg = ok.make_config(layers, vocab=77, width=40, eps=3e-4, scale=6.5)
    ok.save_model_dir(str(tmp_path), cfg, ok.make_weights(cfg))
    spec = spec_of(kge, tmp_path)
    assert (spec["model_type"], spec["vocab"], spec["d"], spec["L"]) == ("nosolix", 77, 40, 3) and spec["has_weights"]
    assert abs(spec["eps"] - 3e-4) < 1e-9 and spec["dyt"] and spec["embed_scale"] == 6.5 and not spec["postnorm"]
    a, b, c = spec["layers"]
    assert (a["mixer"], a["width"], a["n_state"], a["decay_rank"], a["conv"], a["mlp"], a["ff"], a["ff_relu2"]) == (8, 26, 9, 5, 3, 1, 34, 1)
    assert (b["mixer"], b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["window"], b["rot_dims"]) == (9, 6, 3, 10, 7, 19, 6)
    assert abs(b["scale"] - 0.41) < 1e-6 and (b["rot_base"], b["rot_factor"], b["rot_low"], b["rot_high"], b["rot_original"]) == (777.0, 3.0, 1.5, 5.0, 100.0)
    assert (b["m_heads"], b["m_vdim"], b["n_state"], b["ssd_groups"], b["out_norm_groups"], b["conv"]) == (8, 3, 11, 4, 6, 5)
    assert (b["mlp"], b["expert_ff"], b["experts"], b["top"], b["router_groups"], b["groups_keep"], b["group_best"], b["router_correction"]) == (2, 9, 12, 5, 4, 2, 2, 1)
    assert (b["expert_limit"], b["router_scale"], b["shared_ff"], b["shared_limit"], b["shared_gate"]) == (1.25, 1.5, 14, 0.5, 1)
    assert c["mlp"] == 0


def test_config_reader_optional_parts(kge, tmp_path):
    """Rotation without scaling or without any, no mask, a router without groups, no shared expert, no embedding scale."""
    p, q = ok.parallel_layer(), ok.parallel_layer()
    p["mixer"]["left"]["rot"].pop("scaling")
    p["mlp"]["router"].pop("groups")
    p["mlp"].pop("shared")
    q["mixer"]["left"]["rot"] = None
    q["mixer"]["left"]["mask"] = None
    cfg = ok.make_config([p, q])
    cfg.pop("embedding")
    with open(tmp_path / "config.json", "w") as fh:
        json.dump(cfg, fh)
    spec = spec_of(kge, tmp_path)
    a, b = spec["layers"]
    assert (a["rot_factor"], a["router_groups"], a["groups_keep"], a["shared_ff"], a["shared_gate"], spec["embed_scale"]) == (0.0, 1, 1, 0, 0, 1.0)
    assert b["rot_dims"] == 0 and b["window"] == 1 << 30


def test_config_reader_refusals(kge, tmp_path):
    L = kge.lib()

    def refused(change, text):
        cfg = ok.make_config([ok.mamba_layer(), ok.parallel_layer()])
        change(cfg["layers"])
        with open(tmp_path / "config.json", "w") as fh:
            json.dump(cfg, fh)
        assert not L.kge_model_open(str(tmp_path).encode())
        assert text in L.kge_last_error(), L.kge_last_error()
    refused(lambda l: l[0].update(type="wkv"), b"unknown layer type")
    refused(lambda l: l[0]["mixer"].update(inner=0), b"mamba1")
    refused(lambda l: l[0]["mixer"].update(state=257), b"mamba1")
    refused(lambda l: l[0]["mixer"].update(conv=17), b"mamba1")
    refused(lambda l: l[0]["mixer"].update(dt_rank=0), b"mamba1")
    refused(lambda l: l[1]["mixer"].pop("right"), b"'left' and 'right'")
    refused(lambda l: l[1]["mixer"]["left"].update(kv_heads=3), b"attention side")
    refused(lambda l: l[1]["mixer"]["left"]["mask"].update(size=0), b"attention side")
    refused(lambda l: l[1]["mixer"]["left"]["rot"].update(dims=3), b"attention side")
    refused(lambda l: l[1]["mixer"]["left"]["rot"]["scaling"].update(factor=0), b"rotary scaling")
    refused(lambda l: l[1]["mixer"]["right"].update(groups=3), b"recurrent side")
    refused(lambda l: l[1]["mixer"]["right"].update(norm_groups=3), b"recurrent side")
    refused(lambda l: l[1]["mixer"]["right"].update(state=300), b"recurrent side")
    refused(lambda l: l[1]["mlp"]["router"]["groups"].update(count=4), b"expert groups")
    refused(lambda l: l[1]["mlp"]["router"].update(top=4), b"expert groups")
    refused(lambda l: l[1]["mlp"]["expert"].update(limit=0), b"limit")
    refused(lambda l: l[1]["mlp"]["shared"].update(limit=-1.0), b"limit")
    refused(lambda l: l[1]["mlp"]["router"].update(identity=1, experts=5), b"identity")


def test_oracle_dynamic_tanh():
    W = {"n": torch.tensor([2.0, -1.0], dtype=ok.DT), "n.b": torch.tensor([0.5, 0.25], dtype=ok.DT), "n.alpha": torch.tensor(0.5, dtype=ok.DT)}
    y = ok.dyt(torch.tensor([[0.0, 4.0]], dtype=ok.DT), W, "n")
    assert torch.allclose(y, torch.tensor([[0.5, 0.25 - math.tanh(2.0)]], dtype=ok.DT))


def test_oracle_frequencies_and_turn():
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 80.0}}
    f = [100.0 ** (-i / 4.0) for i in range(4)]      # wavelengths 6.3, 19.9, 62.8, 198.7 against 20 and 80
    g = ok.frequencies(rot)
    s = (80.0 / (2.0 * math.pi / f[2]) - 1.0) / 3.0
    assert g[0] == f[0] and g[1] == f[1] and abs(g[3] - f[3] / 4.0) < 1e-15 and abs(g[2] - ((1.0 - s) * f[2] / 4.0 + s * f[2])) < 1e-15
    x = torch.randn(6, 2, 10, dtype=ok.DT)
    y = ok.turn(x, rot)
    assert torch.allclose(y.pow(2).sum(-1), x.pow(2).sum(-1)) and torch.equal(y[0], x[0]) and torch.equal(y[:, :, 8:], x[:, :, 8:])
    a = 3 * g[1]      # position 3, pair (1, 5)
    assert torch.allclose(y[3, 1, 1], x[3, 1, 1] * math.cos(a) - x[3, 1, 5] * math.sin(a)) and torch.allclose(y[3, 1, 5], x[3, 1, 5] * math.cos(a) + x[3, 1, 1] * math.sin(a))


def test_oracle_scans_closed_forms():
    """Two tokens of each recurrence; heads that share a group's B and C."""
    u, D = torch.randn(2, 3, dtype=ok.DT), torch.rand(2, 3, dtype=ok.DT)
    A, B, Cm = -torch.rand(3, 4, dtype=ok.DT), torch.randn(2, 4, dtype=ok.DT), torch.randn(2, 4, dtype=ok.DT)
    y, S = ok.selective_scan(u, D, A, B, Cm)
    S0 = (D[0] * u[0])[:, None] * B[0]
    S1 = torch.exp(D[1][:, None] * A) * S0 + (D[1] * u[1])[:, None] * B[1]
    assert torch.allclose(y[0], S0 @ Cm[0]) and torch.allclose(S, S1) and torch.allclose(y[1], S1 @ Cm[1])
    x, b, c = torch.randn(2, 4, 3, dtype=ok.DT), torch.randn(2, 2, 5, dtype=ok.DT), torch.randn(2, 2, 5, dtype=ok.DT)
    a, d = torch.rand(2, 4, dtype=ok.DT), torch.rand(2, 4, dtype=ok.DT)
    y, S = ok.dual_scan(x, b, c, a, d)
    for h in range(4):
        g = h // 2
        S0 = d[0, h] * torch.outer(b[0, g], x[0, h])
        S1 = a[1, h] * S0 + d[1, h] * torch.outer(b[1, g], x[1, h])
        assert torch.allclose(y[0, h], S0.T @ c[0, g]) and torch.allclose(S[h], S1) and torch.allclose(y[1, h], S1.T @ c[1, g])


def test_oracle_short_conv():
    u, w, b = torch.randn(4, 2, dtype=ok.DT), torch.randn(2, 3, dtype=ok.DT), torch.randn(2, dtype=ok.DT)
    y = ok.short_conv(u, w, b)
    assert torch.allclose(y[0], b + w[:, 2] * u[0]) and torch.allclose(y[3], b + w[:, 0] * u[1] + w[:, 1] * u[2] + w[:, 2] * u[3])


def test_oracle_router():
    """Groups judged by the sum of their two best corrected scores; weights from the plain scores, normalised and scaled."""
    P = {"router": torch.eye(6, dtype=ok.DT), "correction": torch.zeros(6, dtype=ok.DT)}
    s = torch.tensor([[0.90, 0.05, 0.10, 0.60, 0.50, 0.20]], dtype=ok.DT)
    h = torch.log(s / (1.0 - s))
    r = {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 2, "keep": 1}}
    chosen, w = ok.route(h, P, r)      # .90 + .10 against .60 + .50: the second group, although the best expert is in the first
    assert chosen.tolist() == [[3, 4]] and torch.allclose(w, torch.tensor([[1.2 / 1.1, 1.0 / 1.1]], dtype=ok.DT))
    P["correction"] = torch.tensor([0.0, 0.3, 0.0, -0.7, -0.9, -0.9], dtype=ok.DT)
    chosen, w = ok.route(h, P, r)      # the correction enters the choice only
    assert chosen.tolist() == [[0, 1]] and torch.allclose(w, torch.tensor([[1.8 / 0.95, 0.1 / 0.95]], dtype=ok.DT))
    P["correction"] = torch.full((6,), -2.0, dtype=ok.DT)      # all choice scores negative: those left out still do not come in
    assert ok.route(h, P, r)[0].tolist() == [[3, 4]]


def test_oracle_one_token():
    """One token: attention returns its own value, the recurrences start from zero; both sides are normed and averaged."""
    cfg = ok.make_config([ok.parallel_layer(mlp=ok.dense_mlp(5))], width=12)
    W = ok.make_weights(cfg, seed=4)
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    a, b = ok.sub(W, "l0.mix.left."), ok.sub(W, "l0.mix.right.")
    x = W["embed"][5] * cfg["embedding"]["scale"]
    h = ok.dyt(x, W, "l0.norm1")
    v = (a["v"] @ h).reshape(2, 6)[[0, 0, 1, 1]].reshape(-1)
    left = a["o"] @ (v * torch.sigmoid(a["g"] @ h))
    I, GN, r = 20, 12, m["right"]
    p = b["in"] @ h
    xbc = ok.silu(b["conv"][:, -1] * p[I:2 * I + 2 * GN] + b["conv.b"])
    u, B, Cm = xbc[:I].reshape(4, 5), xbc[I:I + GN].reshape(2, 6), xbc[I + GN:].reshape(2, 6)
    dt = torch.log1p(torch.exp(p[2 * I + 2 * GN:] + b["dt_bias"]))
    y = torch.stack([dt[k] * (B[k // 2] @ Cm[k // 2]) * u[k] + b["D"][k] * u[k] for k in range(4)]).reshape(-1) * ok.silu(p[:I])
    y = ok.rms(y.reshape(r["norm_groups"], -1), eps).reshape(-1) * b["norm"]
    x = x + 0.5 * (ok.rms(left, eps, a["out"]) + ok.rms(b["o"] @ y, eps, b["out"]))
    x = x + W["l0.mlp.down"] @ torch.relu(W["l0.mlp.up"] @ ok.dyt(x, W, "l0.norm2")) ** 2
    assert torch.allclose(ok.forward(cfg, W, [5])[0], W["head"] @ ok.dyt(x, W, "final.norm"))
