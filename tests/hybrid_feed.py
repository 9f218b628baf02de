"""What the GPU tests of the hybrid designs share: feeding given tokens through Engine.step, and comparing logits."""
import torch

# largest allowed error of a position's logits (rms over the vocabulary, relative to the logits' own rms)
TOL = {torch.float32: 5e-5, torch.bfloat16: 4e-2}
DTYPES = [torch.float32, torch.bfloat16]


class Feed:
    """Feeds given tokens of several requests through Engine.step and collects the logits of every position."""

    def __init__(self, eng):
        from blitz_scale_b200.runtime import core
        self.eng, self.core = eng, core
        self.batch = core.Batch(0, eng.pool, eng.slots)
        self.got = {}

    def step(self, parts):
        """parts: request number -> its next tokens"""
        for r, toks in parts.items():
            if r in self.batch.request_ids():
                assert self.batch.extend_prompt(r, list(toks))
            else:
                assert self.batch.add_prompts([self.core.SeqSpec(r, list(toks), 1)], False)
                self.got[r] = []
        order = self.batch.request_ids()
        counts = [len(parts.get(r, ())) for r in order]
        logits = self.eng.step(self.batch, counts, [range(n) for n in counts]).cpu()
        at = 0
        for r, n in zip(order, counts):
            self.got[r].append(logits[at:at + n])
            at += n

    def end(self, *requests):
        self.batch.filter([r for r in self.batch.request_ids() if r not in requests])

    def logits(self, r):
        return torch.cat(self.got[r])


def check(got, want, dtype, what=""):
    from blitz_scale_b200 import ops
    ops.check_status()
    assert got.shape == want.shape
    err = ((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt())
    over = int((err > TOL[dtype]).sum())
    # in 16 bits a position may be ill-conditioned (a normalised output close to zero before the norm)
    allowed = max(1, len(err) // 50) if dtype == torch.bfloat16 else 0
    assert over <= allowed and float(err.max()) < 8 * TOL[dtype], (what, "position", int(err.argmax()), float(err.max()), over)
