"""A paged cache with shuffled pages, old rows in them, and the expected attention of a ragged batch."""
import torch

from mindformers_b200.inference.paged_attention import KVCacheContext

from . import gavatar, mefesun


def attention_case(dtype, H, G, D, DV, bs, chunk, lens, news, seed=0, sink_scale=1.0, spots=(), softcap=0.0, score_scale=1.3,
                   device="cuda", window=0, all_values=False):
    """A paged cache with shuffled pages and the step's queries. ``spots``: (sequence, query position, key position) whose
    score is made to stand out (it decides the row where it is visible, and nothing where it is hidden). With ``softcap`` the scores
    are capped and there is no sink, as with ``all_values`` (every head's weights on the values of every KV head)."""
    B = len(lens)
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // bs) for n in lens]
    width = max(per) + 2
    total = sum(per) + 3
    perm = torch.randperm(total, generator=g).tolist()
    ctx = KVCacheContext(1, total, bs, 0, 0, dtype, device, layer_shapes=[(G, D, DV)])
    table = torch.full((B, width), -1, dtype=torch.int32)
    scale = score_scale * D ** -0.5
    qs, ks, vs = [], [], []
    for b in range(B):
        for i in range(per[b]):
            table[b, i] = perm.pop()
        k = torch.randn(lens[b], G, D, generator=g)
        v = torch.randn(lens[b], G, DV, generator=g)
        q = torch.randn(news[b], H, D, generator=g)
        for sb, qp, kp in spots:
            if sb == b:
                r = qp - (lens[b] - news[b])
                k[kp] = q[r].view(G, H // G, D).mean(1) * 6
        qs.append(q.to(dtype)); ks.append(k.to(dtype)); vs.append(v.to(dtype))
    stale = torch.randn(ctx.key_cache[0].shape, generator=g).to(dtype)           # pages hold other requests' old rows
    ctx.key_cache[0].copy_(stale * 5)
    ctx.value_cache[0].copy_(torch.randn(ctx.value_cache[0].shape, generator=g).to(dtype) * 5)
    for b in range(B):
        for t in range(lens[b]):
            at = (int(table[b, t // bs]), t % bs)
            ctx.key_cache[0][at] = ks[b][t].to(device)
            ctx.value_cache[0][at] = vs[b][t].to(device)
    sink = torch.randn(H, generator=g) * sink_scale + 1
    want = []
    for b in range(B):
        n, m = lens[b], news[b]
        reps = H // G
        s = torch.einsum("qhd,khd->hqk", qs[b].double(), ks[b].double().repeat_interleave(reps, 1)) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        mask = mefesun.chunk_mask(n, chunk if chunk else n)[n - m:]
        if window:
            mask = mask & gavatar.window_mask(n, window)[n - m:]
        none = softcap or all_values
        p = mefesun.softmax_with_sink(s, mask, sink.double() if not none else torch.full((H,), -1e30, dtype=torch.float64))
        if all_values:
            want.append(torch.einsum("hqk,kgd->qhgd", p, vs[b].double()))
        else:
            want.append(torch.einsum("hqk,khd->qhd", p, vs[b].double().repeat_interleave(reps, 1)))
    return ctx, table, qs, sink, scale, torch.cat(want).reshape(sum(news), -1)
