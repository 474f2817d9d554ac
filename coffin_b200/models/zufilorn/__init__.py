"""Zufilorn: learned positions, hyper-connected fp32 streams, and layers that mix tokens with a per-channel gated
delta rule, an mLSTM matrix memory or differential attention, in any order."""
