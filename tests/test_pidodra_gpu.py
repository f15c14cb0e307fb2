"""Pidodra on the GPU: every mechanism alone against the plain implementation
(`plain_pidodra`), then whole models through the engine under every way of
cutting the work, and generation through the entry point."""

import math

import numpy as np
import pytest
import torch

import pidodra_models as pm
import plain_pidodra as pp
from test_kegasun_gpu import i32, ops, relerr
from test_zelinex_gpu import _paged_kv
from test_zivulix_gpu import batch_of, f32, tol

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def position_spec(kind, dims, base, head=None, **params):
    from reflex_b200.config.spec import PositionSpec

    return PositionSpec(kind, head or dims, dims, base, tuple(params.items()))


def rotation_of(spec, dtype=torch.float32):
    from reflex_b200.parts.registry import POSITIONS

    return POSITIONS.get(spec.kind)(spec, dtype, DEV).rotation()


def frequencies(rot):
    """rot: (base, dims) or (base, dims, (factor, original, fast, slow))."""
    if len(rot) == 2:
        return pp.inverse_frequencies(rot[1], rot[0]), 1.0
    return pp.yarn_frequencies(rot[1], rot[0], *map(float, rot[2])), pp.yarn_magnitude(rot[2][0])


def spec_of_rot(rot, head):
    if len(rot) == 2:
        return position_spec("rope_neox", rot[1], rot[0], head)
    return position_spec("rope_yarn", rot[1], rot[0], head, **dict(zip(("factor", "original", "fast", "slow"), map(float, rot[2]))))


# ------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("R,H", [(1, 64), (3, 100), (5, 4096), (70, 72), (2, 20000), (4, 33), (6, 6000)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norm_of_the_sum_of_stream_and_result(R, H, out_dtype):
    g = torch.Generator().manual_seed(R + H)
    x, y = torch.randn(R, H, generator=g) * 2, torch.randn(R, H, generator=g) * 5
    w = torch.rand(H, generator=g) + 0.5
    new = pp.rms_norm(1.75 * x.double().numpy() + y.double().numpy(), w.double().numpy(), 1e-3)
    xd = x.to(DEV)
    out = ops().sum_norm(y.to(DEV), xd, 1.75, w.to(DEV), 0.0, 1e-3, out_dtype)
    assert relerr(xd, new) < 3e-6 and out.dtype == out_dtype and relerr(out, new) < tol(out_dtype)
    xd = x.to(DEV)  # a weight stored around zero; no rows asked for
    assert ops().sum_norm(y.to(DEV), xd, 1.75, w.to(DEV) - 1.0, 1.0, 1e-3, None) is None and relerr(xd, new) < 3e-6


@pytest.mark.parametrize("R,H,top", [(1, 64, 1), (5, 100, 3), (40, 2048, 4), (3, 33, 2), (2, 9000, 2)])
@pytest.mark.parametrize("rows_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("weighted", [True, False])
def test_norm_of_the_sum_with_the_experts_weighted_sum_made_on_the_way(R, H, top, rows_dtype, weighted):
    g = torch.Generator().manual_seed(R + H)
    x, yg = torch.randn(R, H, generator=g), (torch.randn(R * top, H, generator=g) * 3).to(rows_dtype)
    place, wts = torch.randperm(R * top, generator=g).to(torch.int32), torch.rand(R, top, generator=g)
    w = torch.rand(H, generator=g) + 0.5
    rows = ops().ExpertRows(yg.to(DEV), place.to(DEV), wts.to(DEV) if weighted else None, R, top)
    f = wts.double().numpy() if weighted else np.ones((R, top))
    y = np.einsum("rk,rkh->rh", f, yg.double().numpy()[place.numpy()].reshape(R, top, H))
    assert relerr(rows.summed(), y) < 3e-6
    xd = x.to(DEV)
    new = pp.rms_norm(0.6 * x.double().numpy() + y, w.double().numpy(), 1e-5)
    out = ops().sum_norm(rows, xd, 0.6, w.to(DEV), 0.0, 1e-5, torch.bfloat16)
    assert relerr(xd, new) < 3e-6 and relerr(out, new) < 8e-3


@pytest.mark.parametrize("E,top,groups", [(16, 4, (4, 2)), (12, 3, (4, 3)), (40, 5, (8, 2)), (100, 7, (10, 1)), (256, 9, (64, 5)),
                                          (5, 1, (5, 2)), (6, 6, None), (96, 40, (3, 2)), (64, 3, (2, 1)), (33, 4, None)])
@pytest.mark.parametrize("R", [1, 7, 64, 300])
def test_experts_chosen_among_the_best_groups(E, top, groups, R):
    """Ids, weights (the softmax over all experts, as it is) and, for up to 64 rows, the
    pairs' places made in the same launch; a row of ties goes to the lower indices."""
    g = torch.Generator().manual_seed(E + R)
    logits = torch.randn(R, E + 3, generator=g) * 2
    logits[-1] = 0.5
    z = logits.double().numpy()[:, 2:2 + E]
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s /= s.sum(axis=1, keepdims=True)
    grp = {"count": groups[0], "keep": groups[1]} if groups else None
    place = R <= ops().MOE_PLACE_MAX_ROWS
    ids, wts, *placed = ops().moe_route(logits.to(DEV), None, top, experts=E, scores="softmax", col0=2, scale=1.75,
                                        groups=groups, place=place)
    ids, wts = ids.cpu().numpy(), wts.cpu().double().numpy()
    for r in range(R):
        want = pp.choose_experts(s[r], top, grp)
        assert ids[r].tolist() == want, r
        assert np.abs(wts[r] - 1.75 * s[r, want]).max() < 1e-6
    if groups and groups[1] < groups[0] and groups[1] < top:
        free = [pp.choose_experts(s[r], top, None) for r in range(R)]
        assert R < 64 or any(f != i for f, i in zip(free, ids.tolist()))   # the groups matter
    if place:
        offsets, at = (t.cpu().numpy() for t in placed[0])
        flat = ids.reshape(-1)
        assert offsets.tolist() == [int((flat < e).sum()) for e in range(E + 1)]
        assert sorted(at.tolist()) == list(range(R * top))
        assert all(offsets[e] <= p < offsets[e + 1] for e, p in zip(flat, at))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("R,E,top,ff,W,groups", [(1, 5, 2, 24, 64, None), (9, 12, 3, 40, 72, (4, 2)), (70, 8, 1, 16, 104, (2, 1)),
                                                 (200, 6, 2, 64, 128, (3, 2)), (5, 40, 4, 21, 50, (8, 3)), (33, 16, 4, 32, 64, (4, 2))])
def test_mixture_of_experts_part(dtype, R, E, top, ff, W, groups):
    """The part alone, its sum made by itself and left to the norm that follows."""
    from reflex_b200.config.spec import FeedForwardSpec
    from reflex_b200.parts.moe import MixtureOfExperts

    g = torch.Generator().manual_seed(E + top + R)
    spec = FeedForwardSpec("moe", hidden_size=W, intermediate_size=ff, params=(
        ("experts", E), ("top", top), ("activation", "swiglu"), ("scores", "softmax"), ("score_scale", 1.3), ("groups", groups)))
    part = MixtureOfExperts(spec, dtype, DEV)
    t = {"router": torch.randn(E, W, generator=g) * 0.4}
    for e in range(E):
        t[f"expert_gate#{e}"] = torch.randn(ff, W, generator=g) * 0.3
        t[f"expert_up#{e}"] = torch.randn(ff, W, generator=g) * 0.3
        t[f"expert_down#{e}"] = torch.randn(W, ff, generator=g) * 0.3
    t = {k: v.to(dtype).float() for k, v in t.items()}
    part.bind(dict(t))
    names = {"expert_gate": "gate", "expert_up": "up", "expert_down": "down"}
    wn = {"router": t["router"].double().numpy()}
    for k, v in t.items():
        if "#" in k:
            role, e = k.split("#")
            wn[f"e{e}.{names[role]}"] = v.double().numpy()
    x = torch.randn(R, W, generator=g).to(dtype)
    mlp = {"router": {"experts": E, "top": top, "scale": 1.3,
                      "groups": {"count": groups[0], "keep": groups[1]} if groups else None}}
    ref = pp.experts_ff(x.double().numpy(), wn, mlp)
    assert relerr(part.forward(x.to(DEV)), ref) < tol(dtype, 1e-5, 1.5e-2)
    left = part.forward(x.to(DEV), leave_sum=True)
    grouped = dtype == torch.bfloat16 and R >= ops().MOE_GROUPED_MIN_ROWS
    assert isinstance(left, ops().ExpertRows) == grouped
    h = torch.randn(R, W, generator=g)
    hd = h.to(DEV)
    ops().sum_norm(left, hd, 1.2, torch.ones(W, device=DEV), 0.0, 1e-6, None)
    assert relerr(hd, pp.rms_norm(1.2 * h.double().numpy() + ref, np.ones(W), 1e-6)) < tol(dtype, 1e-5, 1.5e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,d,dv,rot", [
    (6, 3, 16, 24, (100.0, 8, (4.0, 64, 8.0, 1.0))), (5, 1, 22, 12, (30.0, 6)), (4, 2, 64, 32, (10000.0, 64, (8.0, 256, 16.0, 1.0))),
    (3, 3, 10, 10, (20.0, 2)), (3, 1, 200, 96, (1000.0, 48)), (2, 1, 32, 48, None)])
@pytest.mark.parametrize("writes", [True, False])
def test_norm_then_rotation_and_the_cache_write(dtype, nq, nkv, d, dv, rot, writes):
    """Positions far out, at a page's edge and at zero; heads stored in rows of the
    larger size with zeros behind them; rows without keys and values store nothing."""
    g = torch.Generator().manual_seed(nq + d)
    pos = [0, 1, 63, 64, 65, 1000, 4099]
    R, pad = len(pos), (max(d, dv) + 15) // 16 * 16
    cols = (nq + nkv) * d + nkv * dv if writes else nq * d
    proj = torch.randn(R, (cols + 7) // 8 * 8, generator=g) * 2
    qw, kw = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) + 0.5
    rotation = rotation_of(spec_of_rot(rot, d), dtype) if rot else None
    n_pages = 4099 // 64 + 1
    table = torch.arange(n_pages, dtype=torch.int32).flip(0).reshape(1, n_pages).contiguous()
    kp = torch.full((n_pages, nkv, 64, pad), 7.0, dtype=dtype, device=DEV)
    vp = torch.full((n_pages, nkv, 64, pad), 7.0, dtype=dtype, device=DEV)
    q, _ = ops().rot_qkv_post(proj.to(DEV), None, rotation, None, None, None, False, i32(pos), i32([0] * R), kp, vp,
                              table.to(DEV), 64, nq, nkv, d, dv, pad, writes, dtype,
                              norms=(qw.to(DEV), kw.to(DEV) if writes else None, 1e-5, 0.0))
    x, P = proj.double().numpy()[:, :cols], np.array(pos)
    f, mag = frequencies(rot) if rot else ([], 1.0)

    def made(a, w, n):
        return pp.rotate_halves(pp.rms_norm(a.reshape(R, n, d), w.double().numpy(), 1e-5), P, f, mag)

    t = 3e-4 if dtype == torch.float32 else 8e-3   # 32-bit angles of thousands of radians
    q = q.reshape(R, nq, pad)
    assert relerr(q[..., :d], made(x[:, :nq * d], qw, nq)) < t and float(q[..., d:].abs().sum()) == 0.0
    if not writes:
        assert bool((kp == 7.0).all()) and bool((vp == 7.0).all())
        return
    kr = made(x[:, nq * d:(nq + nkv) * d], kw, nkv)
    v = x[:, (nq + nkv) * d:].reshape(R, nkv, dv)
    for r, p in enumerate(pos):
        page = int(table[0, p // 64])
        assert relerr(kp[page, :, p % 64, :d], kr[r]) < t and relerr(vp[page, :, p % 64, :dv], v[r]) < tol(dtype, 1e-6), p
        assert float(kp[page, :, p % 64, d:].abs().sum()) == 0.0 and float(vp[page, :, p % 64, dv:].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("q_rank,rank,rot,width", [(40, 24, 8, 48), (15, 18, 4, 32), (96, 64, 64, 128), (160, 288, 32, 320),
                                                   (9, 7, 2, 16), (700, 512, 64, 576)])
def test_query_latents_and_cached_rows(dtype, q_rank, rank, rot, width):
    g = torch.Generator().manual_seed(q_rank + rank)
    pos = [0, 5, 63, 64, 999, 4099]
    R, cols = len(pos), q_rank + rank + rot
    proj = torch.randn(R, (cols + 5 + 7) // 8 * 8, generator=g) * 2
    qw, kw = torch.rand(q_rank, generator=g) + 0.5, torch.rand(rank, generator=g) + 0.5
    n_pages = 4099 // 64 + 1
    table = torch.arange(n_pages, dtype=torch.int32).flip(0).reshape(1, n_pages).contiguous()
    pages = torch.full((n_pages, 1, 64, width), float("nan"), dtype=dtype, device=DEV)
    cq = ops().latent_low_post(proj.to(DEV), qw.to(DEV), kw.to(DEV), 1e-5, rotation_of(position_spec("rope_neox", rot, 500.0), dtype),
                               i32(pos), i32([0] * R), pages, table.to(DEV), 64, q_rank, rank, rot, width, True, dtype)
    x = proj.double().numpy()
    assert relerr(cq, pp.rms_norm(x[:, :q_rank], qw.double().numpy(), 1e-5)) < tol(dtype)
    c = pp.rms_norm(x[:, q_rank:q_rank + rank], kw.double().numpy(), 1e-5)
    kr = pp.rotate_halves(x[:, None, q_rank + rank:cols], np.array(pos), pp.inverse_frequencies(rot, 500.0))[:, 0]
    for r, p in enumerate(pos):
        row = pages[int(table[0, p // 64]), 0, p % 64]
        assert relerr(row[:rank], c[r]) < tol(dtype)
        assert relerr(row[rank:rank + rot], kr[r]) < (3e-4 if dtype == torch.float32 else 8e-3)
        assert float(row[rank + rot:].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,n,rot", [(3, 24, 8), (1, 4, 4), (16, 192, 64), (5, 40, 40), (2, 128, 100)])
def test_the_ends_of_heads_turn_where_they_stand(dtype, H, n, rot):
    g = torch.Generator().manual_seed(n + rot)
    pos = [0, 1, 64, 777, 4099]
    x = torch.randn(len(pos), H * n, generator=g).to(dtype)
    out = ops().rotate_tails_(x.to(DEV).clone(), H, rot, rotation_of(position_spec("rope_neox", rot, 1000.0), dtype), i32(pos))
    ref = x.double().numpy().reshape(len(pos), H, n).copy()
    ref[..., n - rot:] = pp.rotate_halves(ref[..., n - rot:], np.array(pos), pp.inverse_frequencies(rot, 1000.0))
    out = out.reshape(len(pos), H, n)
    assert relerr(out, ref) < (3e-4 if dtype == torch.float32 else 8e-3)
    assert torch.equal(out[..., :n - rot].cpu(), x.reshape(len(pos), H, n)[..., :n - rot])


@pytest.mark.parametrize("z_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("R", [3, 16, 20, 90])
def test_per_head_products_with_a_gate_per_element(R, z_dtype):
    g = torch.Generator().manual_seed(R)
    heads, N, K = 3, 40, 24
    x = torch.randn(R, heads * 32, generator=g)
    w = torch.randn(heads, N, K, generator=g) * 0.3
    z = (torch.randn(R, heads * N + 24, generator=g) * 3).to(z_dtype)
    ref = np.einsum("rhk,hnk->rhn", x.double().numpy().reshape(R, heads, 32)[..., :K], w.double().numpy()).reshape(R, -1)
    ref = ref * pp.sigmoid(z.double().numpy()[:, 16:16 + heads * N])
    if z_dtype == torch.float32:
        assert relerr(ops().heads_linear(x.to(DEV), w.to(DEV), gate=(z.to(DEV), 16)), ref) < 1e-5
    xb, wb = x.to(torch.bfloat16), w.to(torch.bfloat16)
    assert relerr(ops().heads_linear(xb.to(DEV), wb.to(DEV), gate=(z.to(DEV), 16)), ref) < 1.5e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("R,heads,n", [(1, 4, 64), (3, 5, 24), (70, 2, 100)])
def test_a_gate_per_head_on_rows(dtype, R, heads, n):
    g = torch.Generator().manual_seed(R)
    a, z = torch.randn(R, heads * n, generator=g).to(dtype), torch.randn(R, heads + 9, generator=g) * 3
    ref = a.double().numpy().reshape(R, heads, n) * pp.sigmoid(z.double().numpy()[:, 5:5 + heads, None])
    assert relerr(ops().sigmoid_gate_mul_(a.to(DEV), z.to(DEV), 5, heads=heads).reshape(R, heads, n), ref) < tol(dtype)


GATE_CASES = [  # nq, nkv, d, [(start, n_new)]
    (6, 3, 32, [(0, 70), (130, 3), (0, 1)]), (8, 2, 128, [(0, 150), (200, 40)]), (8, 4, 64, [(0, 200), (63, 2), (133, 3)]),
    (5, 1, 48, [(0, 140)]), (16, 2, 128, [(500, 1), (63, 1), (64, 1), (0, 1)]), (12, 1, 64, [(300, 1), (700, 1)])]


@pytest.mark.parametrize("kernel", ["plain_f32", "plain_bf16", "prefill_mma", "prefill_tc", "decode", "decode_cluster", "decode_combine"])
@pytest.mark.parametrize("nq,nkv,d,seqs", GATE_CASES)
def test_a_gate_per_head_in_every_attention_kernel(kernel, nq, nkv, d, seqs):
    dtype = torch.float32 if kernel.endswith("f32") else torch.bfloat16
    if kernel == "prefill_tc" and d not in (64, 128):
        pytest.skip("the tcgen05 kernel takes heads of 64 and 128")
    if kernel.startswith("decode") and any(n != 1 for _, n in seqs):
        seqs = [(s + n - 1, 1) for s, n in seqs]
    g = torch.Generator().manual_seed(nq * 100 + d)
    slots, table, kp, vp, ks, vs = _paged_kv([s + n for s, n in seqs], nkv, d, d, dtype, g)
    R = sum(n for _, n in seqs)
    q = torch.randn(R, nq, d, generator=g).to(dtype)
    z = torch.randn(R, nq + 8, generator=g) * 2
    zd = z.to(torch.bfloat16 if kernel == "prefill_tc" else torch.float32).to(DEV)
    scale, ref, r = 2.0 / math.sqrt(d), [], 0
    for (start, n), k, v in zip(seqs, ks, vs):
        kk, vv = k.to(dtype).double().numpy(), v.to(dtype).double().numpy()
        for t in range(n):
            i = start + t + 1
            for h in range(nq):
                s = kk[:i, h // (nq // nkv)] @ q[r, h].double().numpy() * scale
                e = np.exp(s - s.max())
                ref.append((e / e.sum()) @ vv[:i, h // (nq // nkv)] * pp.sigmoid(float(zd[r, 3 + h])))
            r += 1
    ref = np.stack(ref).reshape(R, nq, d)
    b = batch_of(seqs, slots)
    args = (q.reshape(R, nq * d).to(DEV), kp.to(DEV), vp.to(DEV), table.to(DEV), 64)
    if kernel.startswith("decode"):
        n_splits = {"decode": 1, "decode_cluster": 4, "decode_combine": 3}[kernel]
        out = ops().attention_decode(*args, b.row_pos, b.row_slot, nq, nkv, d, None, scale, n_splits=n_splits, gate=(zd, 3))
    elif kernel == "prefill_tc":
        out = ops().attention_prefill_tc(*args, b.seq_slot, b.seq_start, b.seq_new, b.seq_row0, b.max_new, nq, nkv, d, None,
                                         scale, gate=(zd, 3))
    elif kernel == "prefill_mma":
        out = ops().attention_prefill(*args, b.seq_slot, b.seq_start, b.seq_new, b.seq_row0, b.max_new, nq, nkv, d, None, scale)
        out = ops().sigmoid_gate_mul_(out, zd, 3, heads=nq)
    else:
        b.is_decode = False
        out = ops().attention_plain(*args, b.row_pos, b.row_slot, nq, nkv, d, None, scale)
        out = ops().sigmoid_gate_mul_(out, zd, 3, heads=nq)
    ops().check_device_errors(DEV)
    assert relerr(out.reshape(R, nq, d), ref) < tol(dtype, 2e-5, 1.5e-2)
    picked = ops().attention(*args, b, nq, nkv, d, None, scale, gate=(zd, 3))  # whichever kernel the step takes
    assert relerr(picked.reshape(R, nq, d), ref) < tol(dtype, 2e-5, 1.5e-2)


def walk(part, entry_spec, x, dtype, cuts, cache=None, writes=True, slot=None):
    """The mixer over the framework's own cache, in steps of the given sizes."""
    from reflex_b200.cache.store import Cache

    class Ctx:
        shared, state = {}, None

    T = x.shape[0]
    cache = cache or Cache({0: entry_spec}, 1024, 1 << 20, dtype, torch.device(DEV))
    slot = cache.take_slot() if slot is None else slot
    at, step, got = 0, 0, []
    while at < T:
        n = min(cuts[min(step, len(cuts) - 1)], T - at)
        if writes:
            cache.reserve([(slot, n)])
        ctx = Ctx()
        ctx.batch, ctx.kv, ctx.writes_cache = batch_of([(at, n)], [slot]), cache.kv(0), writes
        got.append(part.forward(x[at:at + n].to(dtype).to(DEV).contiguous(), ctx).cpu().double().numpy())
        if writes:
            cache.commit([(slot, n)])
        at, step = at + n, step + 1
    return np.concatenate(got), cache, slot


@pytest.mark.parametrize("H,d,rot,dv,q_rank,rank", [(3, 16, 8, 24, 40, 24), (5, 6, 4, 10, 15, 18), (4, 128, 64, 128, 96, 64),
                                                    (16, 32, 32, 48, 160, 288), (20, 24, 16, 40, 32, 48), (2, 40, 24, 64, 48, 512),
                                                    (2, 100, 20, 96, 36, 600), (6, 48, 16, 32, 64, 80)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_attention_under_every_way_of_cutting(H, d, rot, dv, q_rank, rank, dtype):
    """The mixer without its output product: whole, in portions down to two tokens
    and token by token; the key at position 3 stands out, so queries hundreds of
    positions and several pages later depend on it; sinks of all sizes."""
    from reflex_b200.config.spec import MixerSpec
    from reflex_b200.parts.latent_attention import LatentAttention

    g = torch.Generator().manual_seed(H * 10 + d)
    W, T = 40, 210
    m = {"heads": H, "dim": d, "rot_dim": rot, "vdim": dv, "kv_rank": rank, "scale": 0.5 / math.sqrt(d + rot),
         "rot": {"base": 3000.0, "dims": rot}}
    spec = MixerSpec("latent_attention", hidden_size=W, num_heads=H, num_kv_heads=1, head_dim=d, v_head_dim=dv,
                     scale=m["scale"], position=position_spec("rope_neox", rot, 3000.0, pairing="consecutive"),
                     params=(("q_rank", q_rank), ("kv_rank", rank), ("rot_dim", rot), ("eps", 1e-5), ("sink", True),
                             ("gate", "element")))
    part = LatentAttention(spec, dtype, DEV)
    t = {"q_down": torch.randn(q_rank, W, generator=g) * 0.3, "q_norm": torch.rand(q_rank, generator=g) + 0.5,
         "q_up": torch.randn(H * (d + rot), q_rank, generator=g) * 2.0 / math.sqrt(q_rank), "kv_down": torch.randn(rank + rot, W, generator=g) * 0.3,
         "kv_norm": torch.rand(rank, generator=g) + 0.5, "k_up": torch.randn(H * d, rank, generator=g) / math.sqrt(rank),
         "v_up": torch.randn(H * dv, rank, generator=g) / math.sqrt(rank), "gate": torch.randn(H * dv, W, generator=g) * 0.3,
         "sink": torch.linspace(-8.0, 6.0, H), "o_proj": torch.eye(H * dv)}
    t = {k: v.to(dtype).float() for k, v in t.items()}
    part.bind(dict(t))
    names = {"q_down": "dq", "q_norm": "dq.norm", "q_up": "uq", "kv_down": "dkv", "kv_norm": "dkv.norm", "k_up": "uk", "v_up": "uv",
             "gate": "g", "sink": "sink", "o_proj": "o"}
    w = {names[k]: v.double().numpy() for k, v in t.items()}
    x = torch.randn(T, W, generator=g).to(dtype).float()
    x[3] *= 7.0    # its rotated key part, which is not normed, is seven times as long
    x = x.to(dtype).float()
    ref = pp.latent_attention(x.double().numpy(), w, m, 1e-5)
    without = x.clone()
    without[3] = x[4]
    moved = pp.latent_attention(without.double().numpy(), w, m, 1e-5)
    assert np.abs(ref[-40:] - moved[-40:]).max() > 0.05 * np.abs(ref).max()
    no_sink = pp.latent_attention(x.double().numpy(), dict(w, sink=np.full(H, -99.0)), m, 1e-5)
    assert np.abs(ref - no_sink).max() > 0.05 * np.abs(ref).max()
    cache = None
    for cuts in ([T], [2], [1], [63, 2, 1, 64, 5], [T - 30, 1], [100, 110]):
        got, cache, slot = walk(part, part.cache_spec(), x, dtype, cuts, cache)
        cache.give_slot(slot)
        assert relerr(got, ref) < tol(dtype, 1e-4, 3e-2), cuts
    ops().check_device_errors(DEV)


@pytest.mark.parametrize("H,G,d,dv,rot", [(6, 3, 16, 24, (100.0, 8, (4.0, 64, 8.0, 1.0))), (5, 1, 22, 12, (30.0, 6)),
                                          (8, 2, 128, 128, (10000.0, 96, (8.0, 256, 16.0, 1.0))), (4, 2, 64, 32, (10000.0, 32)),
                                          (4, 4, 40, 40, (500.0, 16)), (3, 3, 10, 10, (20.0, 2)), (2, 1, 32, 80, (50.0, 8))])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_and_a_layer_that_uses_its_keys_and_values(H, G, d, dv, rot, dtype):
    """The mixer without its output product under every way of cutting, and a second
    one with queries, scale and gate of its own over the first one's cache entry.  One key
    stands out: queries anywhere look along a direction that the rotation leaves alone,
    and only the token at position 63 (a page's last) has a key along it."""
    from reflex_b200.config.spec import MixerSpec, NormSpec
    from reflex_b200.parts.attention import GQAttention

    g = torch.Generator().manual_seed(H * 10 + d)
    W, T = 40, 210
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 1.2 / math.sqrt(d),
         "rot": {"base": rot[0], "dims": rot[1], "scaling": dict(zip(("factor", "original", "fast", "slow"), rot[2])) if len(rot) > 2 else None}}
    m2 = dict(m, scale=0.7 / math.sqrt(d))

    def mixer(mm, reads):
        return GQAttention(MixerSpec(
            "gqa_attention", hidden_size=W, num_heads=H, num_kv_heads=G, head_dim=d, v_head_dim=dv, scale=mm["scale"],
            qk_norm=NormSpec("rmsnorm", d, 1e-5), position=spec_of_rot(rot, d),
            params=(("head_gate", True), ("reads_cache", reads))), dtype, DEV)

    def weights(reads):
        t = {"q_proj": torch.randn(H * d, W, generator=g) * 0.3, "q_norm": torch.rand(d, generator=g) + 0.5,
             "g_proj": torch.randn(H, W, generator=g) * 0.3, "o_proj": torch.eye(H * dv)}
        t["q_proj"].view(H, d, W)[:, d - 1, 1] = 6.0      # feature 1 is one everywhere: a query along the last dimension
        if not reads:
            t.update({"k_proj": torch.randn(G * d, W, generator=g) * 0.3, "v_proj": torch.randn(G * dv, W, generator=g) * 0.3,
                      "k_norm": torch.rand(d, generator=g) + 0.5})
            t["k_proj"].view(G, d, W)[:, :, 0] = 0.0
            t["k_proj"].view(G, d, W)[:, d - 1, 0] = 8.0  # feature 0 is set at position 63 alone
        return {k: v.to(dtype).float() for k, v in t.items()}

    names = {"q_proj": "q", "k_proj": "k", "v_proj": "v", "q_norm": "q.norm", "k_norm": "k.norm", "g_proj": "g", "o_proj": "o"}
    t1, t2 = weights(False), weights(True)
    w1, w2 = ({names[k]: v.double().numpy() for k, v in t.items()} for t in (t1, t2))
    first, second = mixer(m, False), mixer(m2, True)
    first.bind(dict(t1))
    second.bind(dict(t2))
    assert set(GQAttention.tensor_specs(second.spec)) == {"q_proj", "o_proj", "g_proj", "q_norm"}
    x, x2 = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g)
    for a in (x, x2):
        a[:, 0], a[:, 1] = 0.0, 1.0
    x[63, 0] = 6.0
    x, x2 = x.to(dtype).float(), x2.to(dtype).float()
    k, v = pp.keys_and_values(x.double().numpy(), w1, m, 1e-5)
    ref = pp.attention(x.double().numpy(), w1, m, 1e-5, k, v)
    ref2 = pp.attention(x2.double().numpy(), w2, m2, 1e-5, k, v)
    vv = v.copy()
    vv[63] = -v[63]
    for a, b in ((ref, pp.attention(x.double().numpy(), w1, m, 1e-5, k, vv)), (ref2, pp.attention(x2.double().numpy(), w2, m2, 1e-5, k, vv))):
        assert np.abs(a[-40:] - b[-40:]).max() > 0.05 * np.abs(a).max() and np.abs(a[:63] - b[:63]).max() < 1e-9
    cache = None
    for cuts in ([T], [2], [1], [63, 2, 1, 64, 5], [T - 30, 1]):
        got, cache, slot = walk(first, first.cache_spec(), x, dtype, cuts, cache)
        assert relerr(got, ref) < tol(dtype, 1e-4, 3e-2), cuts
        got, _, _ = walk(second, None, x2, dtype, cuts, cache, writes=False, slot=slot)
        assert relerr(got, ref2) < tol(dtype, 1e-4, 3e-2), cuts
        cache.give_slot(slot)
    ops().check_device_errors(DEV)


# ----------------------------------------------------------------- whole models
def sharpness(dtype):
    """The full factors in 32-bit, smaller ones in bfloat16 (`pidodra_models.model_folder`)."""
    return True if dtype in ("float32", "f32") else "mild"


def make_engine(name, dtype, max_tokens=4096, **kw):
    import reflex_b200
    from reflex_b200.engine import Engine

    model = reflex_b200.load_model(pm.model_folder(name, sharp=sharpness(dtype)), dtype, DEV)
    return Engine(model, max_tokens=max_tokens, **kw)


_PLAIN = {}


def plain_logits(name, toks, dtype="float32"):
    key = (name, tuple(toks), sharpness(dtype))
    if key not in _PLAIN:
        cfg, w = pp.read_model(pm.model_folder(name, sharp=sharpness(dtype)))
        _PLAIN[key] = pp.forward(cfg, w, toks)
    return _PLAIN[key]


def run_cut(engine, toks, cuts):
    """One sequence fed in steps of the given sizes (the last size repeats)."""
    s = engine.open()
    outs, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        outs.append(engine.step([(s, toks[at:at + n], list(range(n)))]).float().cpu().numpy())
        at += n
        i += 1
    engine.close(s)
    return np.concatenate(outs)


def check_rows(got, ref, dtype, what=""):
    scale = np.abs(ref).max()
    err = np.abs(got - ref).max(axis=1) / scale
    if dtype == "float32":
        assert err.max() < 2e-4, (what, int(err.argmax()), float(err.max()))
    else:
        # bfloat16 rounding moves a close router call now and then: nearly all rows are near
        assert (np.median(err) < 4e-2 or len(err) < 8) and (err > 0.12).sum() <= max(1, 0.05 * len(err)), \
            (what, int(err.argmax()), float(err.max()), float(np.median(err)), int((err > 0.12).sum()))


LENGTHS = {"A": 170, "B": 140, "C": 200, "D": 150, "E": 200}


@pytest.mark.parametrize("name", sorted(pm.ALL))
def test_layer_by_layer_against_the_plain_model(name):
    """The residual after every layer, 32-bit."""
    eng = make_engine(name, "float32")
    toks = pm.tokens(40, pm.ALL[name]["vocab"], 3)
    cfg, w = pp.read_model(pm.model_folder(name))
    ref, seen = [], []
    pp.forward(cfg, w, toks, layers_out=ref)
    eng.model.after_run = lambda i, run, layer, h, pending: seen.append(h.cpu().double().numpy().copy())
    s = eng.open()
    eng.step([(s, toks, [0])])
    eng.close(s)
    eng.model.after_run = None
    assert len(seen) == len(ref) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, ref)):
        assert np.abs(a - b).max() / np.abs(b).max() < 5e-5, (i, np.abs(a - b).max() / np.abs(b).max())


@pytest.mark.parametrize("name", sorted(pm.ALL))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts_and_token_by_token_equal_the_plain_model(name, dtype):
    """Each position's logits, with the prompt in one step, token by token from
    the very first token, and in portions of several sizes down to two tokens:
    every page's edge and the first tokens are met both inside a prompt and in
    decoding."""
    eng = make_engine(name, dtype)
    toks = pm.tokens(LENGTHS[name], pm.ALL[name]["vocab"], 11)
    ref = plain_logits(name, toks, dtype)
    whole = run_cut(eng, toks, [len(toks)])
    check_rows(whole, ref, dtype, "whole")
    for cuts in ([1], [2], [63, 2, 1, 64, 5], [len(toks) - 40, 1]):
        got = run_cut(eng, toks, cuts)
        check_rows(got, ref, dtype, f"cuts {cuts}")
        if dtype == "float32":
            assert np.abs(got - whole).max() / np.abs(ref).max() < 1e-4
    eng.check_errors()


@pytest.mark.parametrize("name", ["A", "C", "E"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batches_in_reused_slots_equal_each_request_alone(name, dtype):
    """Batches of unequal requests, one after another in a small cache, so that
    slots and pages are given back and taken again; shorter requests end early."""
    vocab = pm.ALL[name]["vocab"]
    lens = [1, 70, 3, 131, 64, 9, 200, 2]
    reqs = [pm.tokens(n, vocab, 20 + i) for i, n in enumerate(lens)]
    eng = make_engine(name, dtype, max_tokens=640, max_slots=3, use_graphs=(name != "C"))
    for b0 in range(0, len(reqs), 3):
        idx = list(range(b0, min(len(reqs), b0 + 3)))
        seqs = {i: eng.open() for i in idx}
        fed = {i: 0 for i in idx}
        got = {i: [] for i in idx}
        first = True
        while seqs:
            order = list(seqs)
            entries = []
            for i in order:
                n = max(1, len(reqs[i]) - 20) if first else 1
                part = reqs[i][fed[i]:fed[i] + n]
                entries.append((seqs[i], part, list(range(len(part)))))
            out = eng.step(entries).float().cpu().numpy()
            r = 0
            for i, e in zip(order, entries):
                got[i].append(out[r:r + len(e[1])])
                r += len(e[1])
                fed[i] += len(e[1])
                if fed[i] == len(reqs[i]):
                    eng.close(seqs.pop(i))
            first = False
        for i in idx:
            check_rows(np.concatenate(got[i]), plain_logits(name, reqs[i], dtype), dtype, f"request {i}")
    assert eng.cache.tokens_held() == 0
    eng.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_decoded_tokens_mixed_in_one_step(dtype):
    """One sequence decodes while another brings portions of its prompt, in the same steps."""
    name = "A"
    eng = make_engine(name, dtype)
    vocab = pm.ALL[name]["vocab"]
    a, b = pm.tokens(90, vocab, 31), pm.tokens(150, vocab, 32)
    sa, sb = eng.open(), eng.open()
    got = {sa: [eng.step([(sa, a[:60], list(range(60)))]).float().cpu().numpy()], sb: []}
    at = 0
    for i, n in enumerate([2, 70, 3, 1, 64, 10]):
        out = eng.step([(sa, [a[60 + i]], [0]), (sb, b[at:at + n], list(range(n)))]).float().cpu().numpy()
        got[sa].append(out[:1])
        got[sb].append(out[1:])
        at += n
    check_rows(np.concatenate(got[sa]), plain_logits(name, a, dtype)[:66], dtype, "decoded")
    check_rows(np.concatenate(got[sb]), plain_logits(name, b, dtype), dtype, "portions")


@pytest.mark.parametrize("name", ["A", "C"])
def test_a_wide_batch_of_short_sequences(name):
    """Seventy sequences at once, prompts of a few tokens and then decoded together: more
    rows than the few-row kernels take."""
    eng = make_engine(name, "bfloat16", max_tokens=70 * 64)
    vocab = pm.ALL[name]["vocab"]
    reqs = [pm.tokens(2 + i % 5, vocab, 60 + i) for i in range(70)]
    seqs = [eng.open() for _ in reqs]
    outs = [eng.step([(s, r[:-1], [len(r) - 2]) for s, r in zip(seqs, reqs)]), eng.step([(s, r[-1:], [0]) for s, r in zip(seqs, reqs)])]
    for k, out in enumerate(outs):
        ref = np.stack([plain_logits(name, r, "bfloat16")[len(r) - 2 + k] for r in reqs])
        check_rows(out.float().cpu().numpy(), ref, "bfloat16", f"step {k}")
    eng.check_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_over_many_pages(dtype):
    """A short prompt and 500 decoded tokens over many pages."""
    eng = make_engine("A", dtype, max_tokens=1024)
    toks = pm.tokens(510, pm.ALL["A"]["vocab"], 5)
    ref = plain_logits("A", toks, dtype)
    got = run_cut(eng, toks, [10, 1])
    check_rows(got, ref, dtype, "long decode")
    assert eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_greedy_generation_through_the_entry_point(dtype):
    """`Model.generate` (the scheduler, the sampler, decode graphs in bfloat16)
    against greedy continuation by the plain model."""
    import reflex_b200

    name = "C"
    folder = pm.model_folder(name, sharp=sharpness(dtype))
    model = reflex_b200.Model.load(folder, weights=dtype, max_tokens=2048, max_batch=3)
    vocab = pm.ALL[name]["vocab"]
    prompts = [pm.tokens(n, vocab, 40 + n) for n in (5, 70, 1, 130)]
    n_new = 10
    got = model.generate(prompts, n_new)
    cfg, w = pp.read_model(folder)
    for p, out in zip(prompts, got):
        assert len(out) == n_new
        seq = list(p)
        for t, tok in enumerate(out):
            lg = pp.forward(cfg, w, seq)[-1]
            top2 = np.sort(lg)[-2:]
            if dtype == "bf16" and top2[1] - top2[0] < 0.15 * np.abs(lg).max():
                break  # a near tie: bfloat16 may pick the other one, and the continuations part
            assert tok == int(np.flatnonzero(lg == lg.max())[-1]), (len(p), t)
            seq.append(tok)


@pytest.mark.parametrize("name", ["A", "D"])
def test_decode_steps_are_captured_into_graphs(name):
    eng = make_engine(name, "bfloat16")
    assert eng.model.capturable and eng.use_graphs
