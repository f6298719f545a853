"""Host-side pieces of the Kogonex design: the config reader (every size and constant from config.json, refusals) and
the oracle's own mechanisms against closed forms."""
import ctypes as C
import json
import math

import torch

from oracle import kogonex as ok


def spec_of(kge, path):
    L = kge.lib()
    h = L.kge_model_open(str(path).encode())
    assert h, L.kge_last_error()
    buf = C.create_string_buffer(1 << 16)
    assert L.kge_model_spec_json(h, buf, 1 << 16) > 0
    L.kge_model_close(h)
    return json.loads(buf.value)


def test_config_reader_takes_every_size_and_constant(kge, tmp_path):
    layers = [ok.delta_layer(heads=6, kv_heads=3, dim=5, vdim=7, conv=4, mlp=ok.moe_mlp(ff=9, experts=10, identity=2, top=5, groups=4, keep=2)),
              ok.latent_layer(heads=5, dim=9, rot_dim=6, vdim=11, kv_rank=13, size=19, scale=0.41, base=777.0, factor=3.0, original=100, fast=9.0, slow=2.0, mlp=None),
              ok.latent_layer(heads=2, dim=3, rot_dim=6, vdim=4, kv_rank=13, size=23, scale=0.2, base=777.0, factor=3.0, original=100, fast=9.0, slow=2.0, kv_from=1)]
    cfg = ok.make_config(layers, vocab=77, width=40, eps=3e-4, buckets=101, mul_prev=17, mul_cur=5)
    ok.save_model_dir(str(tmp_path), cfg, ok.make_weights(cfg))
    spec = spec_of(kge, tmp_path)
    assert (spec["model_type"], spec["vocab"], spec["d"], spec["L"]) == ("kogonex", 77, 40, 3) and spec["has_weights"]
    assert abs(spec["eps"] - 3e-4) < 1e-9 and spec["postnorm"] and spec["noprenorm"] and spec["norm_groups"] == 1
    assert (spec["bigram_buckets"], spec["bigram_mul_prev"], spec["bigram_mul_cur"]) == (101, 17, 5)
    a, b, c = spec["layers"]
    assert (a["mixer"], a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["conv"]) == (7, 6, 3, 5, 7, 4)
    assert (a["mlp"], a["expert_ff"], a["experts"], a["identity"], a["top"], a["router_groups"], a["groups_keep"], a["router_correction"]) == (2, 9, 10, 2, 5, 4, 2, 1)
    assert (b["mixer"], b["heads"], b["dim"], b["rot_part"], b["rot_dims"], b["vdim"], b["kv_rank"], b["window"], b["kv_from"]) == (4, 5, 15, 6, 6, 11, 13, 19, -1)
    assert abs(b["scale"] - 0.41) < 1e-6 and (b["rot_base"], b["yarn_factor"], b["yarn_original"], b["yarn_fast"], b["yarn_slow"]) == (777.0, 3.0, 100.0, 9.0, 2.0)
    assert (b["latent_cache"], b["sink"], b["mlp"]) == (1, 1, 0)
    assert (c["heads"], c["dim"], c["vdim"], c["window"], c["kv_from"], c["mlp"]) == (2, 9, 4, 23, 1, 2)


def test_config_reader_optional_parts(kge, tmp_path):
    """Rotation without scaling, a router without groups and identity experts, no bigram table."""
    L = ok.latent_layer()
    L["mixer"]["rot"].pop("scaling")
    L["mlp"]["router"].pop("groups")
    L["mlp"]["router"].pop("identity")
    cfg = ok.make_config([L])
    cfg.pop("embedding")
    with open(tmp_path / "config.json", "w") as fh:
        json.dump(cfg, fh)
    spec = spec_of(kge, tmp_path)
    a = spec["layers"][0]
    assert (a["yarn_factor"], a["router_groups"], a["groups_keep"], a["identity"], spec["bigram_buckets"]) == (0.0, 1, 1, 0, 0)


def test_config_reader_refusals(kge, tmp_path):
    L = kge.lib()

    def refused(change, text):
        cfg = ok.make_config([ok.latent_layer(), ok.delta_layer(), ok.latent_layer(kv_from=0)])
        change(cfg)
        with open(tmp_path / "config.json", "w") as fh:
            json.dump(cfg, fh)
        assert not L.kge_model_open(str(tmp_path).encode())
        assert text in L.kge_last_error(), L.kge_last_error()
    refused(lambda c: c["layers"][0].update(type="wkv"), b"unknown layer type")
    refused(lambda c: c["layers"][1]["mixer"].update(kv_heads=3), b"channel-delta")
    refused(lambda c: c["layers"][1]["mixer"].update(dim=300), b"channel-delta")
    refused(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), b"mask.size")
    refused(lambda c: c["layers"][0]["mixer"].update(kv_rank=0), b"latent-attention")
    refused(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), b"latent-attention")
    refused(lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), b"rotary scaling")
    refused(lambda c: c["layers"][2]["mixer"].update(kv_from=1), b"kv_from")
    refused(lambda c: c["layers"][2]["mixer"].update(kv_from=2), b"kv_from")
    refused(lambda c: c["layers"][2]["mixer"].update(kv_rank=12), b"kv_from")
    refused(lambda c: c["layers"][2]["mixer"]["rot"].update(base=3.0), b"kv_from")
    refused(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), b"expert groups")
    refused(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3), b"expert groups")
    refused(lambda c: c["layers"][0]["mlp"]["router"].update(top=5), b"expert groups")
    refused(lambda c: c["layers"][0]["mlp"].update(kind="dense", ff=8), b"dense")
    refused(lambda c: c["layers"][0]["mlp"].update(shared={"ff": 4}), b"shared")
    refused(lambda c: c["embedding"]["bigram"].update(buckets=0), b"bigram")


def test_oracle_bigram_rows():
    b = {"buckets": 10, "mul_prev": 7, "mul_cur": 3}
    assert ok.bigram_rows([4, 5, 0, 9], b) == [10, (4 * 7 + 15) % 10, (5 * 7) % 10, 27 % 10]


def test_oracle_turn_and_yarn():
    rot = {"base": 100.0, "dims": 4}
    x = torch.randn(6, 4, dtype=ok.DT)
    y = ok.turn(x, list(range(6)), rot)
    assert torch.allclose(y.pow(2).sum(-1), x.pow(2).sum(-1)) and torch.allclose(y[0], x[0])
    a = 3 * 100.0 ** (-2.0 / 4)      # position 3, pair (2, 3)
    assert torch.allclose(y[3, 2], x[3, 2] * math.cos(a) - x[3, 3] * math.sin(a)) and torch.allclose(y[3, 3], x[3, 3] * math.cos(a) + x[3, 2] * math.sin(a))
    # scaling: the fastest pairs keep their frequency, the slowest are divided by the factor, lengths grow by the multiplier
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 6.0, "original": 4096, "fast": 24.0, "slow": 2.0}}
    f, mult = ok.yarn(rot)
    plain = [10000.0 ** (-2.0 * i / 32) for i in range(16)]
    assert f[0] == plain[0] and abs(f[15] - plain[15] / 6.0) < 1e-15 and abs(mult - (0.1 * math.log(6.0) + 1.0)) < 1e-15
    assert all(p / 6.0 <= q <= p for p, q in zip(plain, f)) and any(p / 6.0 < q < p for p, q in zip(plain, f))
    z = torch.randn(3, 32, dtype=ok.DT)
    assert torch.allclose(ok.turn(z, [5, 6, 7], rot).pow(2).sum(-1), mult ** 2 * z.pow(2).sum(-1))


def test_oracle_window_and_sink():
    assert [j for j in range(12) if ok.window_visible(9, j, 3)] == [7, 8, 9]
    s = torch.tensor([[0.0, 1.0, 2.0]], dtype=ok.DT)
    vis = torch.tensor([[False, True, True]])
    w = ok.sink_softmax(s, vis, torch.tensor(0.5, dtype=ok.DT))
    den = math.exp(1.0) + math.exp(2.0) + math.exp(0.5)
    assert torch.allclose(w, torch.tensor([[0.0, math.exp(1.0) / den, math.exp(2.0) / den]], dtype=ok.DT))


def test_oracle_delta_closed_form():
    """Two tokens, one head: the first write is b_0 k_0 v_0^T; the second corrects what the decayed state returns along k_1."""
    q, k = torch.randn(2, 1, 4, dtype=ok.DT), ok.unit(torch.randn(2, 1, 4, dtype=ok.DT))
    v, be, a = torch.randn(2, 1, 3, dtype=ok.DT), torch.rand(2, 1, dtype=ok.DT), torch.rand(2, 1, 4, dtype=ok.DT)
    o, S = ok.delta_scan(q, k, v, be, a)
    S0 = be[0, 0] * torch.outer(k[0, 0], v[0, 0])
    assert torch.allclose(o[0, 0], S0.T @ q[0, 0])
    D = a[1, 0][:, None] * S0
    S1 = D + be[1, 0] * torch.outer(k[1, 0], v[1, 0] - D.T @ k[1, 0])
    assert torch.allclose(S[0], S1) and torch.allclose(o[1, 0], S1.T @ q[1, 0])
    # without decay, a full-strength write makes the state return exactly the value along its (unit) key
    o, S = ok.delta_scan(k, k, v, torch.ones(2, 1, dtype=ok.DT), torch.ones(2, 1, 4, dtype=ok.DT))
    assert torch.allclose(S[0].T @ (k[1, 0] / k[1, 0].norm()), v[1, 0], atol=1e-4)
    # value heads 0, 1 read q / k head 0 and heads 2, 3 head 1
    q2, k2 = torch.randn(3, 2, 4, dtype=ok.DT), torch.randn(3, 2, 4, dtype=ok.DT)
    v2, b2, a2 = torch.randn(3, 4, 2, dtype=ok.DT), torch.rand(3, 4, dtype=ok.DT), torch.rand(3, 4, 4, dtype=ok.DT)
    o2, _ = ok.delta_scan(q2, k2, v2, b2, a2)
    o3, _ = ok.delta_scan(q2[:, 1:], k2[:, 1:], v2[:, 2:3], b2[:, 2:3], a2[:, 2:3])
    assert torch.allclose(o2[:, 2:3], o3)


def test_oracle_router():
    """Groups of neighbours, a correction that enters the choice only, identity experts counted in the groups."""
    P = {"router": torch.eye(6, dtype=ok.DT), "correction": torch.tensor([0.0, 0.0, 0.0, -0.9, 0.0, 0.0], dtype=ok.DT)}
    r = {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 2}}
    h = torch.log(torch.tensor([[0.05, 0.10, 0.15, 0.40, 0.20, 0.10]], dtype=ok.DT))
    chosen, w = ok.route(h, P, r)      # corrected: .05 .10 | .15 -.50 | .20 .10: groups 2 and 1 stay, 4 and 2 are chosen
    assert chosen.tolist() == [[4, 2]] and torch.allclose(w, torch.tensor([[0.20, 0.15]], dtype=ok.DT))
    # all kept choice scores may be negative: the others' still do not come in
    P["correction"] = torch.tensor([-0.5, -0.5, -0.9, -0.9, -0.1, -0.95], dtype=ok.DT)
    chosen, w = ok.route(h, P, dict(r, groups={"count": 3, "keep": 1}))
    assert chosen.tolist() == [[4, 5]] and torch.allclose(w, torch.tensor([[0.20, 0.10]], dtype=ok.DT))
    f = {"expert": {"ff": 3}, "router": r}
    W = {"correction": torch.zeros(6, dtype=ok.DT), "router": P["router"]}
    for e in range(4):
        W.update({f"e{e}.gate": torch.randn(3, 6, dtype=ok.DT), f"e{e}.up": torch.randn(3, 6, dtype=ok.DT), f"e{e}.down": torch.randn(6, 3, dtype=ok.DT)})
    chosen, w = ok.route(h, W, r)      # plain: groups {2, 3} and {4, 5}: 3 and 4
    assert chosen.tolist() == [[3, 4]]
    z = h[0] @ W["e3.gate"].T
    want = 0.40 * ((z * torch.sigmoid(z) * (h[0] @ W["e3.up"].T)) @ W["e3.down"].T) + 0.20 * h[0]
    assert torch.allclose(ok.moe(h, W, f)[0], want)


def test_oracle_one_token_and_layer_sums():
    """One token sees only itself and the sink; a layer adds the normed results to the stream, and the sublayers read the
    stream itself."""
    cfg = ok.make_config([ok.latent_layer(heads=2, dim=3, rot_dim=2, vdim=4, kv_rank=5)], width=8)
    W = ok.make_weights(cfg, seed=4)
    P, eps, m = ok.sub(W, "l0.mix."), cfg["norm"]["eps"], cfg["layers"][0]["mixer"]
    x = W["embed"][5:6] + W["bigram"][53:54]
    z = x @ P["dkv"].T
    c = ok.rms(z[:, :5], eps, P["dkv.norm"])
    q = (x @ P["q"].T).reshape(2, 5)
    k = (c @ P["uk"].T).reshape(2, 3)
    _, mult = ok.yarn(m["rot"])
    s = m["scale"] * ((q[:, :3] * k).sum(-1) + mult ** 2 * (q[:, 3:] * z[0, 5:]).sum(-1))      # position 0: no turn, only the multiplier
    w = torch.exp(s) / (torch.exp(s) + torch.exp(P["sink"]))
    y = ((c @ P["uv"].T).reshape(2, 4) * w[:, None]).reshape(1, 8) @ P["o"].T
    x = x + ok.rms(y, eps, W["l0.norm1"])
    x = x + ok.rms(ok.moe(x, ok.sub(W, "l0.mlp."), cfg["layers"][0]["mlp"]), eps, W["l0.norm2"])
    assert torch.allclose(ok.forward(cfg, W, [5]), ok.rms(x, eps, W["final.norm"]) @ W["head"].T)
