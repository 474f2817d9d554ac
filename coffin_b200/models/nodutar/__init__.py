"""Nodutar: chunked attention beside a gated state in one mixer, attention with distance penalties over its own keys, gated experts,
norms on both sides of every sublayer, layers that run several times."""
