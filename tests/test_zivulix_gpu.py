"""Zivulix on the GPU: every mechanism alone against the plain implementation
(`plain_zivulix`), then whole models through the engine under every way of
cutting the work, and generation through the entry point."""

import math

import numpy as np
import pytest
import torch

import plain_zivulix as pz
import zivulix_models as zm
from test_kegasun_gpu import FakeBatch, i32, ops, relerr
from test_zelinex_gpu import _paged_kv

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def f32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def tol(dtype, exact=3e-6, low=8e-3):
    return exact if dtype == torch.float32 else low


def batch_of(seqs, slots):
    """seqs: (rows already cached, new rows) of each sequence."""
    b = FakeBatch([[0] * n for _, n in seqs], slots, [s for s, _ in seqs])
    b.is_decode = all(n == 1 for _, n in seqs)
    b.max_new = max(n for _, n in seqs)
    b.max_context = max(s + n for s, n in seqs)
    b.starts, b.new_counts = [s for s, _ in seqs], [n for _, n in seqs]
    return b


def rotation_of(base, dims, factor, dtype=torch.float32, head=None):
    from reflex_b200.config.spec import PositionSpec
    from reflex_b200.parts.registry import POSITIONS

    spec = PositionSpec("rope_linear", head or dims, dims, base, (("factor", factor),))
    return POSITIONS.get(spec.kind)(spec, dtype, DEV).rotation()


# ------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("R,H", [(1, 64), (3, 100), (5, 4096), (70, 72), (2, 20000), (4, 33)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norm_on_a_sublayers_result_and_the_next_ones_rows(R, H, out_dtype):
    g = torch.Generator().manual_seed(R + H)
    x, y = torch.randn(R, H, generator=g) * 2, torch.randn(R, H, generator=g) * 5
    w = torch.rand(H, generator=g) - 0.5
    normed = pz.norm_around_zero(y.double().numpy(), w.double().numpy(), 1e-3)
    new = x.double().numpy() + normed
    xd = x.to(DEV)
    out = ops().post_norm(y.to(DEV), xd, w.to(DEV), 1.0, 1e-3, out_dtype)
    assert relerr(xd, new) < 3e-6 and out.dtype == out_dtype and relerr(out, new) < tol(out_dtype)
    xd = x.to(DEV)
    assert ops().post_norm(y.to(DEV), xd, w.to(DEV), 1.0, 1e-3, None) is None and relerr(xd, new) < 3e-6
    yd = y.to(DEV)  # the normed rows alone, in place
    out = ops().post_norm(yd, yd, w.to(DEV), 1.0, 1e-3, out_dtype, fresh=True)
    assert relerr(yd, normed) < 3e-6 and relerr(out, normed) < tol(out_dtype)


@pytest.mark.parametrize("R,groups,gs", [(1, 2, 32), (3, 5, 20), (70, 4, 64), (2, 3, 512), (4, 6, 7)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norm_per_head_with_a_shared_weight_and_a_silu_gate(R, groups, gs, out_dtype):
    g = torch.Generator().manual_seed(R + gs)
    C = groups * gs
    x, w, z = torch.randn(R, C, generator=g) * 3, torch.rand(gs, generator=g) + 0.5, torch.randn(R, C + 24, generator=g) * 3
    ref = (pz.rms_unit(x.double().numpy().reshape(R, groups, gs), 1e-5) * w.double().numpy()).reshape(R, C)
    ref = ref * pz.silu(z.double().numpy()[:, 12:12 + C])
    out = ops().group_norm_gate(x.to(DEV), w.to(DEV), 1e-5, groups, out_dtype, gate=z.to(DEV), gate_col=12,
                                activation="silu")
    assert relerr(out, ref) < tol(out_dtype)


@pytest.mark.parametrize("R,I,K", [(1, 48, 64), (8, 500, 328), (33, 128, 1024), (64, 76, 72), (65, 32, 64), (3, 38, 64),
                                   (5, 125, 200), (4, 20, 100)])
def test_gelu_gated_product_as_epilogue_and_apart(R, I, K):
    """A few bfloat16 rows: the activation rides in the product kernel; more rows, or a
    width that is no multiple of 8: product, then the kernel."""
    g = torch.Generator().manual_seed(R + I)
    x = (torch.randn(R, K, generator=g)).to(torch.bfloat16)
    w = (torch.randn(2 * I, K, generator=g) * 0.3).to(torch.bfloat16)   # rows alternate gate, up
    wn, xn = w.double().numpy(), x.double().numpy()
    ref = pz.gelu_tanh(xn @ wn[0::2].T) * (xn @ wn[1::2].T)
    out = ops().linear_geglu(x.to(DEV), w.to(DEV))
    assert out.dtype == torch.bfloat16 and relerr(out, ref) < 1.5e-2
    assert relerr(ops().linear_geglu(x.float().to(DEV), w.float().to(DEV)), ref) < 1e-5


def test_gelu_far_out_on_both_sides():
    z = torch.tensor([[-60.0, 2.0, -9.0, 2.0, -1.0, 3.0, 0.0, 5.0, 1.0, 1.0, 9.0, 1.0, 60.0, 2.0, 300.0, -1.0]])
    for dtype in (torch.float32, torch.bfloat16):
        out = ops().swiglu(z.to(dtype).to(DEV), alternating=True, activation="gelu_tanh").float().cpu()
        ref = pz.gelu_tanh(z.double().numpy()[:, 0::2]) * z.double().numpy()[:, 1::2]
        assert torch.isfinite(out).all() and relerr(out, ref) < tol(dtype, 1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,d,dv,rot,mix", [
    (6, 3, 16, 24, (100.0, 8, 2.0), "mix"), (5, 1, 22, 12, (30.0, 6, 1.0), None), (8, 2, 128, 128, (10000.0, 64, 4.0), "mix"),
    (2, 1, 64, 32, (10000.0, 64, 3.0), "first"), (4, 4, 20, 20, None, "mix"), (3, 1, 200, 96, (1000.0, 48, 16.0), "first")])
def test_rotation_then_unit_norm_biases_mixed_values_and_the_cache_write(dtype, nq, nkv, d, dv, rot, mix):
    """Positions far out, at a page's edge and at zero; heads stored in rows of the
    larger size with zeros behind them."""
    g = torch.Generator().manual_seed(nq + d)
    pos = [0, 1, 63, 64, 65, 1000, 4099]
    R, pad = len(pos), (max(d, dv) + 15) // 16 * 16
    cols = (nq + nkv) * d + nkv * dv
    proj = torch.randn(R, (cols + 7) // 8 * 8, generator=g) * 2
    bias = torch.randn(cols, generator=g)
    first = torch.randn(R, nkv * dv, generator=g) * 2
    rotation = rotation_of(rot[0], rot[1], rot[2], dtype, d) if rot else None
    n_pages = 4099 // 64 + 1
    table = torch.arange(n_pages, dtype=torch.int32).flip(0).reshape(1, n_pages).contiguous()
    kp = torch.full((n_pages, nkv, 64, pad), float("nan"), dtype=dtype, device=DEV)
    vp = torch.full((n_pages, nkv, 64, pad), float("nan"), dtype=dtype, device=DEV)
    q, kept = ops().rot_qkv_post(
        proj.to(DEV), bias.to(DEV), rotation, 1e-5, f32([0.3]) if mix == "mix" else None,
        first.to(DEV) if mix == "mix" else None, mix == "first", i32(pos), i32([0] * R), kp, vp, table.to(DEV), 64, nq,
        nkv, d, dv, pad, True, dtype)
    x = proj.double().numpy()[:, :cols] + bias.double().numpy()
    dims, base, div = (rot[1], rot[0], rot[2]) if rot else (0, 1.0, 1.0)
    P = np.array(pos)
    qr = pz.rms_unit(pz.rotate(x[:, :nq * d].reshape(R, nq, d), P, dims, base, div), 1e-5)
    kr = pz.rms_unit(pz.rotate(x[:, nq * d:(nq + nkv) * d].reshape(R, nkv, d), P, dims, base, div), 1e-5)
    v = x[:, (nq + nkv) * d:].reshape(R, nkv, dv)
    if mix == "mix":
        vm = 0.7 * v + 0.3 * first.double().numpy().reshape(R, nkv, dv)
    else:
        vm = v
    assert (kept is not None) == (mix == "first")
    if kept is not None:
        assert relerr(kept.reshape(R, nkv, dv), v) < 1e-6
    # 32-bit angles: at position 4,099 an angle of thousands of radians is known to a few 1e-4 of one
    t = 3e-4 if dtype == torch.float32 else 8e-3
    q = q.reshape(R, nq, pad)
    assert relerr(q[..., :d], qr) < t and float(q[..., d:].abs().sum()) == 0.0
    for r, p in enumerate(pos):
        page = int(table[0, p // 64])
        assert relerr(kp[page, :, p % 64, :d], kr[r]) < t, p
        assert relerr(vp[page, :, p % 64, :dv], vm[r]) < tol(dtype, 1e-6), p
        assert float(kp[page, :, p % 64, d:].abs().sum()) == 0.0 and float(vp[page, :, p % 64, dv:].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,rot,rank,width", [(3, 16, 8, 40, 48), (5, 6, 4, 18, 32), (4, 64, 16, 112, 128),
                                                (16, 32, 32, 288, 320), (2, 7, 2, 9, 16)])
def test_latent_rows_with_a_shared_rotated_part_into_the_cache(dtype, H, d, rot, rank, width):
    g = torch.Generator().manual_seed(H + d)
    pos = [0, 5, 63, 64, 999, 4099]
    R = len(pos)
    cols = H * (d + rot) + rank + rot
    proj = torch.randn(R, (cols + 7) // 8 * 8, generator=g) * 2
    w = torch.rand(rank, generator=g) + 0.5
    n_pages = 4099 // 64 + 1
    table = torch.arange(n_pages, dtype=torch.int32).flip(0).reshape(1, n_pages).contiguous()
    pages = torch.full((n_pages, 1, 64, width), float("nan"), dtype=dtype, device=DEV)
    flat, qa = ops().latent_rot_post(proj.to(DEV), w.to(DEV), 1e-5, rotation_of(500.0, rot, 1.0, dtype), i32(pos),
                                     i32([0] * R), pages, table.to(DEV), 64, H, d, rot, rank, width, True, dtype)
    x = proj.double().numpy()
    q = x[:, :H * (d + rot)].reshape(R, H, d + rot)
    down = x[:, H * (d + rot):cols]
    c = pz.rms_unit(down[:, :rank], 1e-5) * w.double().numpy()
    t = 3e-4 if dtype == torch.float32 else 8e-3
    assert relerr(flat.reshape(R, H, d), q[..., :d]) < tol(dtype, 1e-7)
    qa = qa.reshape(R, H, width)
    assert relerr(qa[..., rank:rank + rot], pz.rotate(q[..., d:], np.array(pos), rot, 500.0)) < t
    assert float(qa[..., rank + rot:].abs().sum()) == 0.0
    kr = pz.rotate(down[:, None, rank:], np.array(pos), rot, 500.0)[:, 0]
    for r, p in enumerate(pos):
        row = pages[int(table[0, p // 64]), 0, p % 64]
        assert relerr(row[:rank], c[r]) < tol(dtype) and relerr(row[rank:rank + rot], kr[r]) < t
        assert float(row[rank + rot:].abs().sum()) == 0.0


@pytest.mark.parametrize("R", [3, 20, 90])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_per_head_products_between_rows_of_other_widths(R, dtype):
    """The first K elements of each head of a wider row, into the first N of a wider one."""
    g = torch.Generator().manual_seed(R)
    heads, N, K, xh, yh = 3, 40, 24, 32, 48
    x = torch.randn(R, heads * xh, generator=g).to(dtype)
    w = (torch.randn(heads, N, K, generator=g) * 0.3).to(dtype)
    out = torch.full((R, heads * yh), 7.0, dtype=dtype, device=DEV)
    ops().heads_linear(x.to(DEV), w.to(DEV), out=out)
    ref = np.einsum("rhk,hnk->rhn", x.double().numpy().reshape(R, heads, xh)[..., :K], w.double().numpy())
    out = out.reshape(R, heads, yh)
    assert relerr(out[..., :N], ref) < tol(dtype, 1e-5, 1e-2) and bool((out[..., N:] == 7.0).all())


def capped_ref(q, ks, vs, seqs, scale, window, cap, dtype):
    outs, r = [], 0
    for (start, n), k, v in zip(seqs, ks, vs):
        kk, vv = k.to(dtype).double().numpy(), v.to(dtype).double().numpy()
        for t in range(n):
            i = start + t
            lo = max(0, i - window + 1) if window else 0
            o = np.zeros((q.shape[1], vv.shape[2]))
            for h in range(q.shape[1]):
                kvh = h // (q.shape[1] // kk.shape[1])
                s = (kk[lo:i + 1, kvh] @ q[r + t, h].to(dtype).double().numpy()) * scale
                s = cap * np.tanh(s / cap)
                e = np.exp(s - s.max())
                o[h] = (e / e.sum()) @ vv[lo:i + 1, kvh]
            outs.append(o)
        r += n
    return np.stack(outs)


CAP_CASES = [  # nq, nkv, d, [(start, n_new)], window, cap
    (6, 3, 32, [(0, 70), (130, 3), (0, 1)], 20, 2.0),
    (8, 2, 128, [(0, 150), (200, 40)], 70, 30.0),
    (8, 4, 64, [(0, 200), (63, 2), (133, 3)], 64, 1.5),
    (5, 1, 48, [(0, 140)], None, 3.0),
    (4, 4, 16, [(0, 5), (64, 1), (127, 2)], 1, 4.0),
    (16, 2, 128, [(500, 1), (63, 1), (64, 1), (0, 1)], 200, 2.5),
    (12, 1, 64, [(300, 1), (700, 1)], None, 50.0),
    (4, 1, 240, [(90, 30)], 50, 2.0),
]
CAP_KERNELS = ["plain_f32", "plain_bf16", "prefill_mma", "prefill_tc", "prefill_tc_bound", "decode", "decode_splits"]


def run_capped(kernel, qd, kp, vp, table, batch, nq, nkv, d, window, scale, cap, bound=0.0):
    args = (qd, kp.to(DEV), vp.to(DEV), table.to(DEV), 64)
    if kernel.startswith("plain"):
        return ops().attention_plain(*args, batch.row_pos, batch.row_slot, nq, nkv, d, window, scale, softcap=cap)
    if kernel.startswith("decode"):
        return ops().attention_decode(*args, batch.row_pos, batch.row_slot, nq, nkv, d, window, scale,
                                      n_splits=4 if kernel == "decode_splits" else 1, softcap=cap)
    seq = (batch.seq_slot, batch.seq_start, batch.seq_new, batch.seq_row0, batch.max_new)
    if kernel == "prefill_mma":
        return ops().attention_prefill(*args, *seq, nq, nkv, d, window, scale, softcap=cap)
    return ops().attention_prefill_tc(*args, *seq, nq, nkv, d, window, scale, softcap=cap, score_bound=bound)


@pytest.mark.parametrize("kernel", CAP_KERNELS)
@pytest.mark.parametrize("nq,nkv,d,seqs,window,cap", CAP_CASES)
def test_capped_scores_over_a_window_in_every_attention_kernel(kernel, nq, nkv, d, seqs, window, cap):
    dtype = torch.float32 if kernel.endswith("f32") else torch.bfloat16
    if kernel.startswith("prefill_tc") and d not in (64, 128):
        pytest.skip("the tcgen05 kernel takes heads of 64 and 128")
    if kernel.startswith("decode") and any(n != 1 for _, n in seqs):
        seqs = [(s + n - 1, 1) for s, n in seqs]
    g = torch.Generator().manual_seed(nq * 100 + d)
    slots, table, kp, vp, ks, vs = _paged_kv([s + n for s, n in seqs], nkv, d, d, dtype, g)
    R = sum(n for _, n in seqs)
    q = torch.randn(R, nq, d, generator=g)
    scale = 1.5 / math.sqrt(d)
    bound = 0.0
    if kernel == "prefill_tc_bound":
        # queries and keys of known length: no score beyond half the cap
        q = torch.nn.functional.normalize(q, dim=-1) * math.sqrt(d)
        kmax = max(float(k.norm(dim=-1).max()) for k in ks)
        scale = 0.45 * cap / (math.sqrt(d) * kmax)
        bound = 0.46 * cap
    ref = capped_ref(q, ks, vs, seqs, scale, window, cap, dtype)
    out = run_capped(kernel, q.to(dtype).reshape(R, nq * d).to(DEV), kp, vp, table, batch_of(seqs, slots), nq, nkv, d,
                     window, scale, cap, bound)
    assert relerr(out.reshape(R, nq, d), ref) < tol(dtype, 2e-5, 1.5e-2)


@pytest.mark.parametrize("kernel", CAP_KERNELS[:-1])
@pytest.mark.parametrize("window", [77, None])
def test_a_key_that_stands_out_far_away_and_at_the_windows_edges(kernel, window):
    """Every score is about zero but the one of the key at position 100, capped at 12:
    e^12 against a few hundred ones.  Queries up to position 100 + window - 1 find its
    value, the next one does not; without a window even the last one does."""
    dtype = torch.float32 if kernel.endswith("f32") else torch.bfloat16
    nq, nkv, d, T = 4, 2, 64, 420
    g = torch.Generator().manual_seed(9)
    k = torch.randn(T, nkv, d, generator=g) * 0.02
    v = torch.randn(T, nkv, d, generator=g)
    k[100] = 0.0
    k[100, :, 3] = 8.0
    v[100] = 50.0
    q = torch.randn(T, nq, d, generator=g) * 0.02
    q[:, :, 3] = 8.0     # 64 against the one key before the cap, about zero against the others
    n_pages = (T + 63) // 64
    table = torch.arange(n_pages, dtype=torch.int32).flip(0).reshape(1, n_pages).contiguous()
    kp, vp = torch.zeros(n_pages, nkv, 64, d), torch.zeros(n_pages, nkv, 64, d)
    for p in range(T):
        kp[int(table[0, p // 64]), :, p % 64] = k[p]
        vp[int(table[0, p // 64]), :, p % 64] = v[p]
    W = window or 320
    for i in (99, 100, 101, 100 + W - 2, 100 + W - 1, min(100 + W, T - 1), T - 1):
        if kernel.startswith("decode"):
            seqs = [(i, 1)]
        else:
            seqs = [(max(0, i - 40), min(i, 40) + 1)]   # the query is the last row of a portion
        s, n = seqs[0]
        out = run_capped(kernel, q[s:s + n].to(dtype).reshape(n, nq * d).to(DEV), kp.to(dtype), vp.to(dtype), table,
                         batch_of(seqs, [0]), nq, nkv, d, window, 0.25, 12.0, 16.5)
        seen = float(out.float().reshape(n, nq, d)[-1].abs().max())
        inside = 100 <= i and (window is None or i <= 100 + window - 1)
        assert (seen > 45.0) == inside and (inside or seen < 5.0), (i, seen)




@pytest.mark.parametrize("H,d,rot,dv,rank", [(3, 16, 8, 24, 40), (5, 6, 4, 10, 18), (4, 64, 16, 32, 112), (16, 32, 32, 48, 288),
                                             (20, 24, 16, 40, 48), (3, 128, 64, 128, 256), (2, 40, 24, 64, 512),
                                             (2, 100, 20, 96, 600)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_attention_absorbed_equals_keys_and_values_per_head(H, d, rot, dv, rank, dtype):
    """The mixer without its output product over the framework's own cache: whole, in
    portions down to two tokens and token by token; the key at position 3 stands out,
    so queries hundreds of positions and several pages later depend on it."""
    from reflex_b200.cache.store import Cache
    from reflex_b200.config.spec import MixerSpec, PositionSpec
    from reflex_b200.parts.latent_attention import LatentAttention

    g = torch.Generator().manual_seed(H * 10 + d)
    W, T = 40, 210
    m = {"heads": H, "dim": d, "rot_dim": rot, "vdim": dv, "kv_rank": rank, "scale": 0.3 / math.sqrt(d + rot),
         "rot": {"base": 300.0, "dims": rot}}
    spec = MixerSpec("latent_attention", hidden_size=W, num_heads=H, num_kv_heads=1, head_dim=d, v_head_dim=dv,
                     scale=m["scale"], position=PositionSpec("rope_neox", rot, rot, 300.0),
                     params=(("kv_rank", rank), ("rot_dim", rot), ("eps", 1e-5)))
    part = LatentAttention(spec, dtype, DEV)
    t = {"q_proj": torch.randn(H * (d + rot), W, generator=g) * 0.3, "kv_down": torch.randn(rank + rot, W, generator=g) * 0.3,
         "kv_norm": torch.rand(rank, generator=g) + 0.5, "k_up": torch.randn(H * d, rank, generator=g) * 0.3,
         "v_up": torch.randn(H * dv, rank, generator=g) * 0.3, "o_proj": torch.eye(H * dv)}
    t = {k: v.to(dtype).float() for k, v in t.items()}
    part.bind(dict(t))
    names = {"q_proj": "q", "kv_down": "dkv", "kv_norm": "dkv.norm", "k_up": "uk", "v_up": "uv", "o_proj": "o"}
    x = torch.randn(T, W, generator=g).to(dtype).float()
    x[3] *= 12.0    # its rotated key part, which is not normed, is twelve times as long
    x = x.to(dtype).float()
    ref = pz.latent_attention(x.double().numpy(), {names[k]: v.double().numpy() for k, v in t.items()}, m, 1e-5)
    without = x.clone()
    without[3] = x[4]
    moved = pz.latent_attention(without.double().numpy(), {names[k]: v.double().numpy() for k, v in t.items()}, m, 1e-5)
    assert np.abs(ref[-40:] - moved[-40:]).max() > 0.05 * np.abs(ref).max()
    cache = Cache({0: part.cache_spec()}, 1024, 1 << 20, dtype, torch.device(DEV))

    class Ctx:
        writes_cache, shared = True, {}

    for cuts in ([T], [2], [63, 2, 1, 64, 5], [T - 30, 1]):
        slot, at, step, got = cache.take_slot(), 0, 0, []
        while at < T:
            n = min(cuts[min(step, len(cuts) - 1)], T - at)
            cache.reserve([(slot, n)])
            ctx = Ctx()
            ctx.batch, ctx.kv, ctx.state = batch_of([(at, n)], [slot]), cache.kv(0), None
            got.append(part.forward(x[at:at + n].to(dtype).to(DEV).contiguous(), ctx).cpu().double().numpy())
            cache.commit([(slot, n)])
            at, step = at + n, step + 1
        cache.give_slot(slot)
        assert relerr(np.concatenate(got), ref) < tol(dtype, 1e-4, 3e-2), cuts


@pytest.mark.parametrize("H,G,d,dv,taps", [(4, 2, 16, 24, 4), (2, 1, 10, 7, 1), (1, 1, 33, 50, 3), (4, 2, 128, 64, 4),
                                           (2, 2, 72, 160, 3), (6, 2, 32, 16, 2), (2, 1, 64, 128, 4), (1, 1, 300, 12, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_delta_rule_carried_through_its_state(H, G, d, dv, taps, dtype):
    """The mixer without its output product, two sequences side by side in slots of a
    state tensor that held other numbers before: whole, token by token, two tokens at a
    time and in unequal steps (some shorter than the filters look back)."""
    from reflex_b200.config.spec import MixerSpec
    from reflex_b200.parts.gated_delta import GatedDelta

    g = torch.Generator().manual_seed(H * 10 + d)
    W = 40
    spec = MixerSpec("gated_delta", hidden_size=W, num_heads=H, num_kv_heads=G, head_dim=d, v_head_dim=dv, scale=d ** -0.5,
                     params=(("taps", taps), ("unit_eps", 1e-6), ("eps", 1e-5)))
    part = GatedDelta(spec, dtype, DEV)
    t = {"q_proj": torch.randn(G * d, W, generator=g) * 0.4, "k_proj": torch.randn(G * d, W, generator=g) * 0.4,
         "v_proj": torch.randn(H * dv, W, generator=g) * 0.4, "g_proj": torch.randn(H * dv, W, generator=g) * 0.3,
         "b_proj": torch.randn(H, W, generator=g) * 0.3, "a_proj": torch.randn(H, W, generator=g) * 0.3,
         "q_conv": torch.rand(G * d, taps, generator=g) * 1.2 - 0.6, "k_conv": torch.rand(G * d, taps, generator=g) * 1.2 - 0.6,
         "v_conv": torch.rand(H * dv, taps, generator=g) * 1.2 - 0.6, "A_log": torch.rand(H, generator=g) - 3.0,
         "dt_bias": torch.rand(H, generator=g) - 0.5, "norm": torch.rand(dv, generator=g) + 0.5, "o_proj": torch.eye(H * dv)}
    t = {k: v.to(dtype).float() for k, v in t.items()}      # what both sides see
    part.bind(dict(t))
    names = {"q_proj": "q", "k_proj": "k", "v_proj": "v", "g_proj": "g", "b_proj": "b", "a_proj": "a", "q_conv": "q.conv",
             "k_conv": "k.conv", "v_conv": "v.conv", "A_log": "A_log", "dt_bias": "dt_bias", "norm": "norm", "o_proj": "o"}
    wn = {names[k]: v.double().numpy() for k, v in t.items()}
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv}
    lens = [47, 90]
    xs = [torch.randn(n, W, generator=g).to(dtype).float() for n in lens]
    refs = [pz.delta_mixer(x.double().numpy(), wn, m, 1e-5) for x in xs]

    class Ctx:
        pass

    for cuts in ([100], [1], [2], [7, 2, 1, 40]):
        state = torch.randn(5, part.cache_spec().shape[0], generator=g).to(DEV)
        state[1].zero_()
        state[3].zero_()
        fed, got, step = [0, 0], [[], []], 0
        while any(f < n for f, n in zip(fed, lens)):
            take = [min(cuts[min(step, len(cuts) - 1)], n - f) for f, n in zip(fed, lens)]
            live = [i for i in range(2) if take[i] > 0]
            ctx = Ctx()
            ctx.batch = batch_of([(fed[i], take[i]) for i in live], [[3, 1][i] for i in live])
            ctx.state = state
            rows = torch.cat([xs[i][fed[i]:fed[i] + take[i]] for i in live]).to(dtype).to(DEV).contiguous()
            y = part.forward(rows, ctx).cpu().double().numpy()
            r = 0
            for i in live:
                got[i].append(y[r:r + take[i]])
                r += take[i]
                fed[i] += take[i]
            step += 1
        for i in range(2):
            assert relerr(np.concatenate(got[i]), refs[i]) < tol(dtype, 1e-4, 3e-2), (cuts, i)


@pytest.mark.parametrize("exact", [True, False])
def test_a_slow_decay_keeps_a_far_write_and_a_write_rate_of_one_replaces_it(exact):
    """One head: a value written under one key is read 400 tokens later when the decay is
    one and other tokens write under another key; it is gone after one write under the
    same key at a rate of one, and after one token with a decay of zero."""
    d, dv, T = 8, 16, 401
    for what in ("kept", "replaced", "decayed"):
        q, k, v = np.zeros((T, d)), np.zeros((T, d)), np.zeros((T, dv))
        q[:, 0] = 1.0
        k[:, 1] = 1.0
        k[0] = 0.0
        k[0, 0] = 1.0
        v[0, 2] = 7.0
        decay, rate = np.ones((T, 1)), np.ones((T, 1))
        if what == "replaced":
            k[200] = k[0]
        if what == "decayed":
            decay[200] = 0.0
        state = torch.zeros(1, dv * d, device=DEV)
        o = ops().gated_delta_scan(f32(np.concatenate([q, k, v], axis=1)), f32(np.concatenate([decay, rate], axis=1)),
                                   state, 0, batch_of([(0, T)], [0]), 1, 1, d, dv, exact=exact).cpu().numpy()
        assert abs(o[0, 2] - 7.0) < 1e-5 and abs(o[199, 2] - 7.0) < 1e-5
        assert abs(o[-1, 2] - (7.0 if what == "kept" else 0.0)) < 1e-5, what


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 64, 64), (3, 3, 24, 16), (6, 2, 128, 128), (2, 1, 96, 48), (1, 1, 256, 32),
                                      (2, 2, 200, 80)])
def test_sixteen_rows_at_a_time_equal_the_row_by_row_walk(H, G, d, dv):
    """Sequences of lengths around the chunks' edges beside one another, states that are not
    zero at the start, strong and weak decays: both kernels against the plain recurrence,
    and far closer to it than products of rounded operands would be."""
    g = torch.Generator().manual_seed(H + d)
    lens = [8, 15, 16, 17, 33, 1, 100]
    R, n = sum(lens), len(lens)
    q, k = torch.randn(R, G, d, generator=g), torch.randn(R, G, d, generator=g)
    k[20:30] = k[20:21]    # the same key many times within a chunk
    q, k = torch.nn.functional.normalize(q, dim=-1), torch.nn.functional.normalize(k, dim=-1)
    v = torch.randn(R, H, dv, generator=g)
    decay, rate = torch.rand(R, H, generator=g) ** 0.2, torch.rand(R, H, generator=g)
    decay[5], decay[40] = 1e-12, 1.0
    rate[22:26] = 1.0
    S0 = torch.randn(n, H, dv, d, generator=g)
    qkv = torch.cat([q.reshape(R, -1), k.reshape(R, -1), v.reshape(R, -1)], dim=1).to(DEV)
    gates = torch.cat([decay, rate], dim=1).to(DEV)
    refs, ends, r = [], [], 0
    for i, m in enumerate(lens):
        S = S0[i].double().numpy().transpose(0, 2, 1).copy()
        for t in range(r, r + m):
            o = np.zeros((H, dv))
            for h in range(H):
                kt, qt = k[t, h // (H // G)].double().numpy(), q[t, h // (H // G)].double().numpy()
                S[h] = float(decay[t, h]) * S[h]
                S[h] += np.outer(kt, float(rate[t, h]) * (v[t, h].double().numpy() - S[h].T @ kt))
                o[h] = S[h].T @ qt
            refs.append(o.reshape(-1))
        ends.append(S.transpose(0, 2, 1))
        r += m
    for exact in (True, False):
        state = torch.cat([torch.full((n, 4), 3.0), S0.reshape(n, -1)], dim=1).to(DEV).contiguous()
        o = ops().gated_delta_scan(qkv, gates, state, 4, batch_of([(0, m) for m in lens], list(range(n))), H, G, d, dv,
                                   exact=exact)
        assert relerr(o, np.stack(refs)) < 5e-6, exact
        assert relerr(state[:, 4:].reshape(n, H, dv, d), np.stack(ends)) < 5e-6 and bool((state[:, :4] == 3.0).all())


def test_a_layer_that_mixes_values_needs_the_first_ones():
    from reflex_b200.config.spec import MixerSpec
    from reflex_b200.errors import InvalidInput
    from reflex_b200.parts.capped_attention import CappedAttention

    spec = MixerSpec("capped_attention", hidden_size=16, num_heads=1, num_kv_heads=1, head_dim=16, scale=1.0,
                     params=(("unit_eps", 1e-5), ("value_mix", "mix")))
    part = CappedAttention(spec, torch.float32, DEV)

    class Ctx:
        writes_cache, shared, kv, batch = True, {}, None, None

    with pytest.raises(InvalidInput):
        part.forward(torch.zeros(1, 16, device=DEV), Ctx())


# ----------------------------------------------------------------- whole models
def sharpness(dtype):
    """The full factors in 32-bit; their square roots in bfloat16 (`zivulix_models.model_folder`)."""
    return True if dtype in ("float32", "f32") else "mild"


def make_engine(name, dtype, max_tokens=4096, **kw):
    import reflex_b200
    from reflex_b200.engine import Engine

    model = reflex_b200.load_model(zm.model_folder(name, sharp=sharpness(dtype)), dtype, DEV)
    return Engine(model, max_tokens=max_tokens, **kw)


_PLAIN = {}


def plain_logits(name, toks, dtype="float32"):
    key = (name, tuple(toks), sharpness(dtype))
    if key not in _PLAIN:
        cfg, w = pz.read_model(zm.model_folder(name, sharp=sharpness(dtype)))
        _PLAIN[key] = pz.forward(cfg, w, toks)
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
        assert (np.median(err) < 4e-2 or len(err) < 8) and (err > 0.12).sum() <= max(1, 0.05 * len(err)), \
            (what, int(err.argmax()), float(err.max()), float(np.median(err)))


LENGTHS = {"A": 170, "B": 140, "C": 200, "D": 150, "E": 300}


@pytest.mark.parametrize("name", sorted(zm.ALL))
def test_layer_by_layer_against_the_plain_model(name):
    """The residual after every layer, 32-bit."""
    eng = make_engine(name, "float32")
    toks = zm.tokens(40, zm.ALL[name]["vocab"], 3)
    cfg, w = pz.read_model(zm.model_folder(name))
    ref, seen = [], []
    pz.forward(cfg, w, toks, layers_out=ref)
    eng.model.after_run = lambda i, run, layer, h, pending: seen.append(h.cpu().double().numpy().copy())
    s = eng.open()
    eng.step([(s, toks, [0])])
    eng.close(s)
    eng.model.after_run = None
    assert len(seen) == len(ref) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, ref)):
        assert np.abs(a - b).max() / np.abs(b).max() < 5e-5, (i, np.abs(a - b).max() / np.abs(b).max())


@pytest.mark.parametrize("name", sorted(zm.ALL))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts_and_token_by_token_equal_the_plain_model(name, dtype):
    """Each position's logits, with the prompt in one step, token by token from
    the very first token, and in portions of several sizes down to two tokens:
    the windows' edges, the filters' look back, every page's edge and the first
    tokens are met both inside a prompt and in decoding."""
    eng = make_engine(name, dtype)
    toks = zm.tokens(LENGTHS[name], zm.ALL[name]["vocab"], 11)
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
    slots, pages and state vectors are given back and taken again; shorter
    requests end early."""
    vocab = zm.ALL[name]["vocab"]
    lens = [1, 70, 3, 131, 64, 9, 200, 2]
    reqs = [zm.tokens(n, vocab, 20 + i) for i, n in enumerate(lens)]
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
    vocab = zm.ALL[name]["vocab"]
    a, b = zm.tokens(90, vocab, 31), zm.tokens(150, vocab, 32)
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_over_many_pages(dtype):
    """A short prompt and 500 decoded tokens: the memories and the filters' last inputs
    are carried for hundreds of steps, the windows pass over decoded tokens many times
    and their pages are given back, the latents' pages stay."""
    eng = make_engine("A", dtype, max_tokens=1024)
    toks = zm.tokens(510, zm.ALL["A"]["vocab"], 5)
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
    folder = zm.model_folder(name, sharp=sharpness(dtype))
    model = reflex_b200.Model.load(folder, weights=dtype, max_tokens=2048, max_batch=3)
    vocab = zm.ALL[name]["vocab"]
    prompts = [zm.tokens(n, vocab, 40 + n) for n in (5, 70, 1, 130)]
    n_new = 10
    got = model.generate(prompts, n_new)
    cfg, w = pz.read_model(folder)
    for p, out in zip(prompts, got):
        assert len(out) == n_new
        seq = list(p)
        for t, tok in enumerate(out):
            lg = pz.forward(cfg, w, seq)[-1]
            top2 = np.sort(lg)[-2:]
            if dtype == "bf16" and top2[1] - top2[0] < 0.15 * np.abs(lg).max():
                break  # a near tie: bfloat16 may pick the other one, and the continuations part
            assert tok == int(np.flatnonzero(lg == lg.max())[-1]), (len(p), t)
            seq.append(tok)


@pytest.mark.parametrize("name", ["A", "D"])
def test_decode_steps_are_captured_into_graphs(name):
    eng = make_engine(name, "bfloat16")
    assert eng.model.capturable and eng.use_graphs


@pytest.mark.parametrize("shape,dtype", [((3,), torch.float32), ((8, 5), torch.float32), ((4096,), torch.float32), ((1,), torch.int32),
                                         ((20000,), torch.float32)])
@pytest.mark.parametrize("n", [1, 3, 70])
def test_the_state_of_chosen_slots_is_copied_aside_and_put_back(shape, dtype, n):
    from reflex_b200.cache.specs import StateSpec
    from reflex_b200.cache.store import StateGroup

    g = torch.Generator().manual_seed(n)
    grp = StateGroup(StateSpec(shape, str(dtype).split(".")[1]), [0, 1, 2], 80, torch.device(DEV))
    grp.data.copy_(torch.randint(-1000, 1000, tuple(grp.data.shape), generator=g).to(dtype))
    slots = torch.randperm(80, generator=g)[:n].tolist()
    before = grp.data.clone()
    saved = grp.snapshot(slots)
    assert torch.equal(saved[1], before[:, slots])
    grp.data.add_(5)
    grp.restore(saved)
    assert torch.equal(grp.data[:, slots], before[:, slots])
    others = [s for s in range(80) if s not in slots]
    assert torch.equal(grp.data[:, others], before[:, others] + 5)
